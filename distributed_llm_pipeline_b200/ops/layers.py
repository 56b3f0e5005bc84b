"""Ops of layer-list models (recurrent mixers, latent attention, norms behind the sublayers): thin wrappers over the C ABI.

There is no CPU form: the kernels are the only implementation.  Two storage types run through every op, bf16 and fp32 (`f32`); the
residual stream, norms, recurrent states, attention scores and weights are fp32 in both.
"""
from __future__ import annotations

import ctypes as C

import torch

from . import api
from . import lib as _lib

OUT_F32, OUT_GEGLU, OUT_BF16 = 0, 1, 2
HGRN2_CHUNK = 64            # tokens per chunk of the chunked recurrence


class RowStage(C.Structure):
    """How a row is formed in front of a product: x (+ gnorm(y) * w1 -> h_out), then optionally gnorm(.) * w2."""
    _fields_ = [("x", C.c_void_p), ("x_f32", C.c_int32), ("ldx", C.c_int32), ("y", C.c_void_p), ("ldy", C.c_int32), ("w1", C.c_void_p),
                ("groups1", C.c_int32), ("h_out", C.c_void_p), ("ldh", C.c_int32), ("w2", C.c_void_p), ("groups2", C.c_int32), ("w2_mod", C.c_int32),
                ("eps", C.c_float), ("K", C.c_int32), ("Kp", C.c_int32)]


class Hgrn2Args(C.Structure):
    _fields_ = [("proj", C.c_void_p), ("ldp", C.c_int32), ("fbias", C.c_void_p), ("lower", C.c_void_p), ("state", C.c_void_p), ("seg", C.c_void_p),
                ("seg_slot", C.c_void_p), ("pos", C.c_void_p), ("out", C.c_void_p), ("ldo", C.c_int32), ("H", C.c_int32), ("D", C.c_int32), ("V", C.c_int32),
                ("n_seg", C.c_int32)]


class Hgrn2Chunks(C.Structure):
    _fields_ = [("chunk", C.c_void_p), ("first", C.c_void_p), ("states", C.c_void_p), ("decay", C.c_void_p), ("n_chunks", C.c_int32), ("pad", C.c_int32)]


class LatentArgs(C.Structure):
    _fields_ = [("q", C.c_void_p), ("cache", C.c_void_p), ("block_table", C.c_void_p), ("tok_slot", C.c_void_p), ("pos", C.c_void_p),
                ("tile_row0", C.c_void_p), ("tile_rows", C.c_void_p), ("out", C.c_void_p), ("part_o", C.c_void_p), ("part_ml", C.c_void_p),
                ("max_pages", C.c_int32), ("page_size", C.c_int32), ("H", C.c_int32), ("Rc", C.c_int32), ("T", C.c_int32), ("n_tiles", C.c_int32),
                ("bm", C.c_int32), ("n_splits", C.c_int32), ("scale", C.c_float)]


def load_library():
    _lib.load_layers()


def _need_cuda(t: torch.Tensor, what: str):
    if not t.is_cuda:
        raise RuntimeError(f"{what}: layer-list models run on a CUDA device only")


def _p(t):
    return None if t is None else t.data_ptr()


def row_stage(x: torch.Tensor, K: int, Kp: int, eps: float, y=None, w1=None, groups1: int = 1, h_out=None, w2=None, groups2: int = 1) -> RowStage:
    return RowStage(_p(x), int(x.dtype == torch.float32), x.stride(0), _p(y), y.stride(0) if y is not None else 0, _p(w1), groups1, _p(h_out),
                    h_out.stride(0) if h_out is not None else 0, _p(w2), groups2, w2.numel() if w2 is not None else 1, eps, K, Kp)


def matvec_fits(T: int, w: torch.Tensor) -> bool:
    """The staged rows and the partial sums fit the shared memory of one block (very wide fp32 rows do not)."""
    return (T if T != 3 else 4) * w.shape[1] * w.element_size() <= 150 * 1024


def matvec(st: RowStage, w: torch.Tensor, out: torch.Tensor, T: int, geglu: bool = False) -> torch.Tensor:
    """1..4 staged rows times w^T, w [N, ld] bf16 or fp32; out fp32 [T, N], or GEGLU of interleaved rows -> activation type [T, N/2]."""
    _need_cuda(w, "matvec")
    _lib.check(_lib.load().dlp_layers_matvec(C.byref(st), _p(w), w.stride(0), w.shape[0], _p(out), out.stride(0), OUT_GEGLU if geglu else OUT_F32, T,
                                             int(w.dtype == torch.float32), api._stream()), "layers_matvec")
    api._count()
    return out


def stage_rows(st: RowStage, xb: torch.Tensor, T: int) -> torch.Tensor:
    _need_cuda(xb, "stage_rows")
    _lib.check(_lib.load().dlp_layers_stage_rows(C.byref(st), _p(xb), xb.stride(0), T, int(xb.dtype == torch.float32), api._stream()), "layers_stage_rows")
    api._count()
    return xb


def linear(x: torch.Tensor, w: torch.Tensor, out: torch.Tensor, geglu: bool = False) -> torch.Tensor:
    """x [T, K] (activation type, K = padded width) times w^T through the tcgen05 GEMM (bf16) or the fp32 kernel."""
    _need_cuda(x, "linear")
    f32 = w.dtype == torch.float32
    mode = OUT_GEGLU if geglu else OUT_F32 if out.dtype == torch.float32 else OUT_BF16
    ws = None if f32 else api.gemm_workspace(x.device)
    _lib.check(_lib.load().dlp_layers_linear(_p(x), x.stride(0), _p(w), w.stride(0), w.shape[0], w.shape[1], _p(out), out.stride(0),
                                             mode, x.shape[0], int(f32), _p(ws), 0 if ws is None else ws.numel(), api._stream()),
               "layers_linear")
    api._count()
    return out


def head_matmul(x: torch.Tensor, x_head: int, kx: int, w: torch.Tensor, N: int, out: torch.Tensor, out_head: int, T: int, gate: torch.Tensor | None = None):
    """out[t, h, :N] = x[t, h * x_head : + kx] . w[h]^T (* sigmoid(gate[t, h])); w [H, rows, Kp] zero-padded along Kp."""
    _need_cuda(w, "head_matmul")
    f32 = w.dtype == torch.float32
    _lib.check(_lib.load().dlp_layers_head_matmul(_p(x), int(x.dtype == torch.float32), x.stride(0), x_head, kx, _p(w), w.shape[2], w.shape[0], N, w.shape[1],
                                                  _p(out), out.stride(0), out_head, _p(gate), gate.stride(0) if gate is not None else 0, T, int(f32),
                                                  api._stream()), "layers_head_matmul")
    api._count()
    return out


def embed(table: torch.Tensor, ids: torch.Tensor, h: torch.Tensor, T: int):
    _need_cuda(table, "embed")
    _lib.check(_lib.load().dlp_layers_embed(_p(table), table.stride(0), _p(ids), _p(h), h.shape[1], T, table.shape[0], int(table.dtype == torch.float32),
                                            api._stream()), "layers_embed")
    api._count()


def latent_write(proj: torch.Tensor, w: torch.Tensor, eps: float, R: int, slot: torch.Tensor, cache: torch.Tensor, T: int):
    """RMS norm of the latent columns `proj` [T, R] (any row stride) into the paged latent cache [..., Rc]."""
    _need_cuda(cache, "latent_write")
    _lib.check(_lib.load().dlp_layers_latent_write(_p(proj), proj.stride(0), _p(w), eps, R, cache.shape[-1], _p(slot), _p(cache), T,
                                                   int(cache.dtype == torch.float32), api._stream()), "layers_latent_write")
    api._count()


def hgrn2(proj: torch.Tensor, fbias, lower, state: torch.Tensor, seg, seg_slot, n_seg: int, pos, out: torch.Tensor, chunks=None):
    """Gated linear recurrence of the listed segments; proj rows are q | f | v before their activations, state [slots, H, D, V], seg
    [n_seg, 2] token ranges.  chunks = (chunk table [n, 2], first chunk of every segment [n_seg + 1], states workspace, decay workspace):
    64-token chunks on the tensor cores (at most 128 channels per head) instead of the token scan."""
    _need_cuda(state, "hgrn2")
    _, H, D, V = state.shape
    a = Hgrn2Args(_p(proj), proj.stride(0), _p(fbias), _p(lower), _p(state), _p(seg), _p(seg_slot), _p(pos), _p(out), out.stride(0), H, D, V, n_seg)
    c = None
    if chunks is not None:
        table, first, states, decay = chunks
        n = table.shape[0]
        if states.numel() < n * H * D * V or decay.numel() < n * H * D:
            raise ValueError("hgrn2: workspace too small")
        c = Hgrn2Chunks(_p(table), _p(first), _p(states), _p(decay), n, 0)
    _lib.check(_lib.load().dlp_layers_hgrn2(C.byref(a), C.byref(c) if c is not None else None, api._stream()), "layers_hgrn2")
    api._count(3 if c is not None else 1)
    return out


def hgrn2_chunk_table(segs: list[tuple[int, int]]) -> tuple[list[int], list[int]]:
    """(first token, length) of every chunk and the first chunk of every segment, for token ranges `segs`."""
    table, first = [], [0]
    for lo, hi in segs:
        for t in range(lo, hi, HGRN2_CHUNK):
            table += [t, min(HGRN2_CHUNK, hi - t)]
        first.append(len(table) // 2)
    return table, first


def latent_tile_rows(H: int, T: int) -> int:
    """(token, head) rows per tile: enough to fill the tensor-core rows, no more than a batch of single tokens has."""
    return 64 if T * H > 4096 or H >= 48 else 32 if H > 16 else 16


def latent_attention(q, cache, block_table, tok_slot, pos, tile_row0, tile_rows, n_tiles: int, bm: int, H: int, T: int, scale: float, out, n_splits: int = 1,
                     workspace=None):
    _need_cuda(cache, "latent_attention")
    po, pm = workspace if workspace is not None and n_splits > 1 else (None, None)
    a = LatentArgs(_p(q), _p(cache), _p(block_table), _p(tok_slot), _p(pos), _p(tile_row0), _p(tile_rows), _p(out), _p(po), _p(pm), block_table.shape[1],
                   cache.shape[-2], H, cache.shape[-1], T, n_tiles, bm, n_splits, scale)
    _lib.check(_lib.load().dlp_layers_latent_attention(C.byref(a), int(cache.dtype == torch.float32), api._stream()), "layers_latent_attention")
    api._count(2 if n_splits > 1 else 1)
    return out


def latent_gather(cache, block_table_row, S: int, out):
    """Latent rows 0 .. S-1 of one request out of its pages -> out [S, Rc] (bf16)."""
    _need_cuda(cache, "latent_gather")
    _lib.check(_lib.load().dlp_layers_latent_gather(_p(cache), _p(block_table_row), cache.shape[-2], cache.shape[-1], _p(out), S, api._stream()), "layers_latent_gather")
    api._count()
    return out


def head_rows(x, H: int, D: int, Dp: int, out):
    """fp32 columns [T, H * D] -> bf16 rows [T, H * Dp], heads padded with zeros."""
    _need_cuda(x, "head_rows")
    _lib.check(_lib.load().dlp_layers_head_rows(_p(x), x.stride(0), D, Dp, H, _p(out), x.shape[0], api._stream()), "layers_head_rows")
    api._count()
    return out


def rows_attention(q, kv, S: int, pos0: int, H: int, Dp: int, Vp: int, V: int, scale: float, out, gate=None):
    """Causal attention of q [T, H * Dp] at positions pos0 .. over kv [S, H * (Dp + Vp)]; out [T, H * V], each head times sigmoid(gate)."""
    _need_cuda(q, "rows_attention")
    _lib.check(_lib.load().dlp_layers_rows_attention(_p(q), _p(kv), kv.stride(0), S, q.shape[0], pos0, H, Dp, Vp, V, scale, _p(gate),
                                                     gate.stride(0) if gate is not None else 0, _p(out), out.stride(0), api._stream()), "layers_rows_attention")
    api._count()
    return out


def check_waits():
    """Raise if a wait inside an attention kernel gave up since the last call (synchronises the device)."""
    flag = C.c_int(0)
    _lib.check(_lib.load().dlp_layers_rows_attention_error(C.byref(flag)), "rows_attention_error")
    if flag.value:
        raise _lib.DlpError("a wait inside the attention kernel ran into its limit")
