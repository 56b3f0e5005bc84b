"""Ops of layer-list models (recurrent mixers, delta rule, latent, windowed and differential attention, routed experts, norms on either side): thin wrappers over the C ABI.

There is no CPU form: the kernels are the only implementation.  Two storage types run through every op, bf16 and fp32 (`f32`); the
residual stream, norms, recurrent states, attention scores and weights are fp32 in both.
"""
from __future__ import annotations

import ctypes as C
from dataclasses import dataclass

import torch

from . import api
from . import lib as _lib

OUT_F32, OUT_GEGLU, OUT_BF16, OUT_RELU2, OUT_SWIGLU = 0, 1, 2, 3, 4       # gated ones take interleaved (gate, up) rows
GATE_SIGMOID_AFTER, GATE_SILU_BEFORE, GATE_SILU_AFTER = 1, 2, 3
MAX_EXPERTS, MAX_TOP = 256, 32
GQA_MMA_DIM, GQA_FLASH_DIM = 256, 128      # widest heads of the tensor-core forms
ROWS_FLASH_KEY, ROWS_FLASH_VALUE = 192, 128     # widest heads of the flash kernel on expanded rows
NO_WINDOW = 1 << 30
FLASH_TILE = 128            # tokens per tile of the tcgen05 flash kernel
HGRN2_CHUNK, SSD_CHUNK, DELTA_CHUNK = 64, 128, 64       # tokens per chunk of the chunked recurrences
SSD_DIM = 256              # widest keys of the chunked and single-token forms of the scalar-decay recurrence
DELTA_DIM = 128            # widest keys of the chunked form of the delta rule
LONG_FROM = 128            # segments from this length on take the chunked recurrences and the expanded / flash attention
CONV_TAPS = 32


class RowStage(C.Structure):
    """How a row is formed in front of a product: x (+ y or gnorm(y) * w1) (+ e) (-> h_out), then optionally gnorm(.) * w2, or with b2 a layer norm.
    Mixer outputs: x1 - lam * x2 of two maps (pair), silu(g) in front of the norm, or sigmoid(g) or silu(g)
    behind it.  tail (mat-vec): values behind the row as they are."""
    _fields_ = [("x", C.c_void_p), ("x_f32", C.c_int32), ("ldx", C.c_int32), ("y", C.c_void_p), ("ldy", C.c_int32), ("w1", C.c_void_p),
                ("groups1", C.c_int32), ("h_out", C.c_void_p), ("ldh", C.c_int32), ("w2", C.c_void_p), ("groups2", C.c_int32), ("w2_mod", C.c_int32),
                ("eps", C.c_float), ("K", C.c_int32), ("Kp", C.c_int32), ("b2", C.c_void_p), ("e", C.c_void_p), ("lde", C.c_int32),
                ("pair", C.c_int32), ("g", C.c_void_p), ("ldg", C.c_int32), ("gate", C.c_int32), ("lam", C.c_float), ("tail", C.c_void_p),
                ("ld_tail", C.c_int32), ("K_tail", C.c_int32)]


class OutTail(C.Structure):
    """Behind a product's sums: a bias, and outputs from n2 on behind xIELU (z / 2 + pos z^2 above zero, z / 2 + neg (exp(z) - 1 - z) below) in the
    activation type to out2."""
    _fields_ = [("bias", C.c_void_p), ("out2", C.c_void_p), ("n2", C.c_int32), ("ldo2", C.c_int32), ("pos", C.c_float), ("neg", C.c_float)]


class RouteRule(C.Structure):
    _fields_ = [("bias", C.c_void_p)] + [(n, C.c_int32) for n in ("n_expert", "top", "sigmoid", "groups", "keep")] + [("scale", C.c_float)]


class ExpertArgs(C.Structure):
    _fields_ = [("logits", C.c_void_p), ("rule", RouteRule), ("w", C.c_void_p)] + [(n, C.c_int32) for n in ("ldl", "rows", "ldw", "act")] + \
               [(n, C.c_void_p) for n in ("w_s", "x_s", "act_s")] + [(n, C.c_int32) for n in ("rows_s", "K_s", "ldw_s", "ldx_s", "ld_act_s")]


@dataclass
class Routing:
    """Which experts a token uses.  softmax: the `top` largest of logits + bias, weighted by the softmax over those.  sigmoid: scores
    sigmoid(logits); the `keep` best of `groups` groups of neighbours (sum of a group's two largest score + bias), the `top` largest of
    score + bias in those, weighted by their scores over the sum of them, times scale."""
    bias: torch.Tensor | None
    n: int
    top: int
    sigmoid: bool = False
    groups: int = 1
    keep: int = 1
    scale: float = 1.0

    def c(self) -> RouteRule:
        return RouteRule(_p(self.bias), self.n, self.top, int(self.sigmoid), self.groups, self.keep, self.scale)


class GqaArgs(C.Structure):
    _fields_ = [(n, C.c_void_p) for n in ("proj", "q_norm", "k_norm", "inv_freq", "q", "kc", "vc", "block_table", "tok_slot", "pos", "slot", "tile_row0", "tile_rows", "out")] + \
               [(n, C.c_int32) for n in ("ldp", "ldo", "T", "H", "G", "D", "V", "Dc", "Vc", "rot", "max_pages", "page_size", "n_pages", "n_tiles", "bm", "n_splits", "window",
                                         "keep", "chunk", "maps", "adjacent")] + [("eps", C.c_float), ("scale", C.c_float), ("rot_scale", C.c_float), ("v_first", C.c_void_p), ("v_mix", C.c_int32), ("v_lam", C.c_float)]


class Hgrn2Args(C.Structure):
    _fields_ = [("proj", C.c_void_p), ("ldp", C.c_int32), ("fbias", C.c_void_p), ("lower", C.c_void_p), ("state", C.c_void_p), ("seg", C.c_void_p),
                ("seg_slot", C.c_void_p), ("pos", C.c_void_p), ("out", C.c_void_p), ("ldo", C.c_int32), ("H", C.c_int32), ("D", C.c_int32), ("V", C.c_int32),
                ("n_seg", C.c_int32)]


class ScanChunks(C.Structure):
    _fields_ = [("chunk", C.c_void_p), ("first", C.c_void_p), ("states", C.c_void_p), ("decay", C.c_void_p), ("n_chunks", C.c_int32), ("pad", C.c_int32)]


class SsdArgs(C.Structure):
    _fields_ = [(n, C.c_void_p) for n in ("q", "k", "v", "decay", "log_decay", "dt", "dt_bias", "skip", "state", "seg", "seg_slot", "pos", "out")] + \
               [(n, C.c_int32) for n in ("ldq", "ldk", "ldv", "rows_f32", "act", "hpg", "lddt", "ldo", "H", "D", "V", "n_seg")]


class DeltaArgs(C.Structure):
    _fields_ = [(n, C.c_void_p) for n in ("q", "k", "v", "a", "b", "log_decay", "dt_bias", "state", "seg", "seg_slot", "pos", "out")] + \
               [(n, C.c_int32) for n in ("ldq", "ldk", "ldv", "rows_f32", "hpg", "lda", "ldb", "ldo", "H", "D", "V", "n_seg")] + [("unit_eps", C.c_float), ("q_scale", C.c_float)]


class DeltaChunks(C.Structure):
    _fields_ = [(n, C.c_void_p) for n in ("chunk", "first", "states", "keys", "solve", "weights", "u", "gates")] + [("n_chunks", C.c_int32), ("pad", C.c_int32)]


class LatentRows(C.Structure):
    _fields_ = [(n, C.c_void_p) for n in ("proj", "w", "slot", "cache", "pos", "inv_freq", "q")] + [(n, C.c_int32) for n in ("ldp", "R", "Rc", "rot", "adjacent", "ldq", "H", "Dq")] + \
               [("eps", C.c_float), ("rot_scale", C.c_float)]


class ConvArgs(C.Structure):
    _fields_ = [(n, C.c_void_p) for n in ("x", "w", "b", "ring")] + [(n, C.c_int32) for n in ("ldx", "taps", "channels")]


class LatentArgs(C.Structure):
    _fields_ = [("q", C.c_void_p), ("cache", C.c_void_p), ("block_table", C.c_void_p), ("tok_slot", C.c_void_p), ("pos", C.c_void_p),
                ("tile_row0", C.c_void_p), ("tile_rows", C.c_void_p), ("out", C.c_void_p), ("part_o", C.c_void_p), ("part_ml", C.c_void_p),
                ("max_pages", C.c_int32), ("page_size", C.c_int32), ("H", C.c_int32), ("Rc", C.c_int32), ("Vc", C.c_int32), ("T", C.c_int32),
                ("n_tiles", C.c_int32), ("bm", C.c_int32), ("n_splits", C.c_int32), ("window", C.c_int32), ("scale", C.c_float)]


def load_library():
    _lib.load_layers()


def _need_cuda(t: torch.Tensor, what: str):
    if not t.is_cuda:
        raise RuntimeError(f"{what}: layer-list models run on a CUDA device only")


def _p(t):
    return None if t is None else t.data_ptr()


def row_stage(x: torch.Tensor, K: int, Kp: int, eps: float, y=None, w1=None, groups1: int = 1, h_out=None, w2=None, groups2: int = 1,
              b2=None, e=None, pair: int = 0, lam: float = 0.0, g=None, gate: int = 0, tail=None) -> RowStage:
    return RowStage(_p(x), int(x.dtype == torch.float32), x.stride(0), _p(y), y.stride(0) if y is not None else 0, _p(w1), groups1, _p(h_out),
                    h_out.stride(0) if h_out is not None else 0, _p(w2), groups2, w2.numel() if w2 is not None else 1, eps, K, Kp, _p(b2), _p(e), e.stride(0) if e is not None else 0,
                    pair, _p(g), g.stride(0) if g is not None else 0, gate, lam, _p(tail), tail.stride(0) if tail is not None else 0, tail.shape[1] if tail is not None else 0)


def out_tail(bias=None, n2: int = (1 << 31) - 1, out2=None, act: tuple[float, float] = (0.0, 0.0)) -> OutTail:
    """act: xIELU's two coefficients."""
    return OutTail(_p(bias), _p(out2), n2, out2.stride(0) if out2 is not None else 0, *act)


def _ref(s):
    return None if s is None else C.byref(s)


def matvec_fits(T: int, w: torch.Tensor) -> bool:
    """The staged rows and the partial sums fit the shared memory of one block (very wide fp32 rows do not)."""
    return (T if T != 3 else 4) * w.shape[1] * w.element_size() <= 150 * 1024


def matvec(st: RowStage, w: torch.Tensor, out: torch.Tensor, T: int, act: int = OUT_F32, tail: OutTail | None = None) -> torch.Tensor:
    """1..4 staged rows times w^T, w [N, ld] bf16 or fp32; out fp32 [T, N] (tail: `out_tail`), or behind an activation (OUT_*) in the activation type
    (gated: [T, N/2])."""
    _need_cuda(w, "matvec")
    _lib.check(_lib.load().dlp_layers_matvec(C.byref(st), _p(w), w.stride(0), w.shape[0], _p(out), out.stride(0), act, _ref(tail), T,
                                             int(w.dtype == torch.float32), api._stream()), "layers_matvec")
    api._count()
    return out


def stage_rows(st: RowStage, xb: torch.Tensor, T: int) -> torch.Tensor:
    _need_cuda(xb, "stage_rows")
    _lib.check(_lib.load().dlp_layers_stage_rows(C.byref(st), _p(xb), xb.stride(0), T, int(xb.dtype == torch.float32), api._stream()), "layers_stage_rows")
    api._count()
    return xb


def linear(x: torch.Tensor, w: torch.Tensor, out: torch.Tensor, act: int = OUT_F32, tail: OutTail | None = None) -> torch.Tensor:
    """x [T, K] (activation type, K = padded width) times w^T through the tcgen05 GEMM (bf16) or the fp32 kernel."""
    _need_cuda(x, "linear")
    f32 = w.dtype == torch.float32
    mode = OUT_BF16 if act == OUT_F32 and out.dtype != torch.float32 and tail is None else act
    ws = None if f32 else api.gemm_workspace(x.device)
    _lib.check(_lib.load().dlp_layers_linear(_p(x), x.stride(0), _p(w), w.stride(0), w.shape[0], w.shape[1], _p(out), out.stride(0),
                                             mode, _ref(tail), x.shape[0], int(f32), _p(ws), 0 if ws is None else ws.numel(), api._stream()),
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


def embed(table: torch.Tensor, ids: torch.Tensor, h: torch.Tensor, T: int, scale: float = 1.0):
    _need_cuda(table, "embed")
    _lib.check(_lib.load().dlp_layers_embed(_p(table), table.stride(0), _p(ids), _p(h), h.shape[1], T, table.shape[0], scale, int(table.dtype == torch.float32),
                                            api._stream()), "layers_embed")
    api._count()


def latent_write(proj: torch.Tensor, w: torch.Tensor, eps: float, R: int, slot: torch.Tensor, cache: torch.Tensor, T: int, rot=None, q=None, heads: int = 0):
    """RMS norm of the latent columns `proj` [T, R] (any row stride) into the paged latent cache [..., Rc].  rot = (positions, frequencies, factor on cosine
    and sine): 2 * len(frequencies) more columns, turned in neighbouring pairs, go behind them, and those at the end of every head of q
    [T, heads * size] (fp32) are turned in place."""
    _need_cuda(cache, "latent_write")
    pos, f, amp = rot if rot is not None else (None, None, 1.0)
    a = LatentRows(_p(proj), _p(w), _p(slot), _p(cache), _p(pos), _p(f), _p(q), proj.stride(0), R, cache.shape[-1], 2 * f.numel() if f is not None else 0, 1,
                   q.stride(0) if q is not None else 0, heads, q.shape[1] // heads if q is not None else 0, eps, amp)
    _lib.check(_lib.load().dlp_layers_latent_write(C.byref(a), T, int(cache.dtype == torch.float32), api._stream()), "layers_latent_write")
    api._count()


def hgrn2(proj: torch.Tensor, fbias, lower, state: torch.Tensor, seg, seg_slot, n_seg: int, pos, out: torch.Tensor, chunks=None):
    """Gated linear recurrence of the listed segments; proj rows are q | f | v before their activations, state [slots, H, D, V], seg
    [n_seg, 2] token ranges.  chunks = (chunk table [n, 2], first chunk of every segment [n_seg + 1], states workspace, decay workspace):
    64-token chunks (HGRN2_CHUNK) on the tensor cores (at most 128 channels per head) instead of the token scan."""
    _need_cuda(state, "hgrn2")
    _, H, D, V = state.shape
    a = Hgrn2Args(_p(proj), proj.stride(0), _p(fbias), _p(lower), _p(state), _p(seg), _p(seg_slot), _p(pos), _p(out), out.stride(0), H, D, V, n_seg)
    c = None
    if chunks is not None:
        table, first, states, decay = chunks
        n = table.shape[0]
        if states.numel() < n * H * D * V or decay.numel() < n * H * D:
            raise ValueError("hgrn2: workspace too small")
        c = ScanChunks(_p(table), _p(first), _p(states), _p(decay), n, 0)
    _lib.check(_lib.load().dlp_layers_hgrn2(C.byref(a), C.byref(c) if c is not None else None, api._stream()), "layers_hgrn2")
    api._count(3 if c is not None else 1)
    return out


def scan_chunk_table(segs: list[tuple[int, int]], size: int) -> tuple[list[int], list[int]]:
    """(first token, length) of every chunk of `size` tokens and the first chunk of every segment, for token ranges `segs`."""
    table, first = [], [0]
    for lo, hi in segs:
        for t in range(lo, hi, size):
            table += [t, min(size, hi - t)]
        first.append(len(table) // 2)
    return table, first


def ssd(rows, heads_per_group: int, state: torch.Tensor, decay, log_decay, seg, seg_slot, n_seg: int, pos, out: torch.Tensor, act: bool = False, steps=None, skip=None, chunks=None,
        conv=None, single: bool = False):
    """Recurrence with one decay per head and token over the listed segments.  rows = (q, k, v): columns of the first head onwards, fp32 or bf16
    (act: silu on the way); state [slots, H, D, V]; steps = (raw step sizes [T, H], their bias): decays exp(log_decay * softplus(.)),
    else the constant `decay`.  chunks as for `hgrn2` (SSD_CHUNK tokens each, workspace for one decay per chunk and head); single: every segment is one token, and with
    conv = `conv_args` of its inputs the rows are the raw columns in front of the convolution."""
    _need_cuda(state, "ssd")
    q, k, v = rows
    _, H, D, V = state.shape
    dt, dt_bias = steps if steps is not None else (None, None)
    a = SsdArgs(_p(q), _p(k), _p(v), _p(decay), _p(log_decay), _p(dt), _p(dt_bias), _p(skip), _p(state), _p(seg), _p(seg_slot), _p(pos), _p(out), q.stride(0), k.stride(0), v.stride(0),
                int(q.dtype == torch.float32), int(act), heads_per_group, dt.stride(0) if dt is not None else 0, out.stride(0), H, D, V, n_seg)
    c = None
    if chunks is not None:
        table, first, states, decays = chunks
        n = table.shape[0]
        if states.numel() < n * H * D * V or decays.numel() < n * H:
            raise ValueError("ssd: workspace too small")
        c = ScanChunks(_p(table), _p(first), _p(states), _p(decays), n, 0)
    _lib.check(_lib.load().dlp_layers_ssd(C.byref(a), C.byref(c) if c is not None else None, C.byref(conv) if conv is not None else None, 1 if c is not None else 2 if single else 0,
                                          api._stream()), "layers_ssd")
    api._count(3 if c is not None else 1)
    return out


def ssd_single_fits(D: int, V: int) -> bool:
    return D <= SSD_DIM and V % 4 == 0


def conv_args(x: torch.Tensor, w: torch.Tensor, b: torch.Tensor | None, ring: torch.Tensor) -> ConvArgs:
    """x [T, channels] fp32 (any row stride), w [taps, channels], b [channels] or None, ring [slots, taps, channels]."""
    return ConvArgs(_p(x), _p(w), _p(b), _p(ring), x.stride(0), w.shape[0], w.shape[1])


def conv_rows(x, w, b, ring, seg, seg_slot, n_seg: int, longest: int, pos, out):
    """Causal convolution per channel and silu over the listed segments -> out [T, channels]; leaves their last inputs in the ring."""
    _need_cuda(ring, "conv_rows")
    c = conv_args(x, w, b, ring)
    _lib.check(_lib.load().dlp_layers_conv_rows(C.byref(c), _p(seg), _p(seg_slot), _p(pos), n_seg, longest, _p(out), out.stride(0), int(out.dtype == torch.float32), api._stream()),
               "layers_conv_rows")
    api._count()
    return out


def delta(rows, heads_per_group: int, state: torch.Tensor, a, b, log_decay, dt_bias, seg, seg_slot, n_seg: int, pos, out: torch.Tensor, unit_eps: float, chunks=None, conv=None,
          single: bool = False):
    """Gated delta rule over the listed segments.  rows = (q, k, v): columns of the first head onwards, fp32 or bf16, behind convolution and activation;
    a, b [T, H]: raw step sizes (decay exp(log_decay * softplus(a + dt_bias))) and raw write strengths; q and k are made unit vectors per head
    (unit_eps inside the root), q is scaled by D^-1/2.  chunks = (chunk table [n, 2], first chunk of every segment [n_seg + 1], workspaces as
    `delta_workspace` lists them): 64-token chunks (DELTA_CHUNK) on the tensor cores; single, conv: as for `ssd`."""
    _need_cuda(state, "delta")
    q, k, v = rows
    _, H, D, V = state.shape
    args = DeltaArgs(_p(q), _p(k), _p(v), _p(a), _p(b), _p(log_decay), _p(dt_bias), _p(state), _p(seg), _p(seg_slot), _p(pos), _p(out), q.stride(0), k.stride(0), v.stride(0),
                     int(q.dtype == torch.float32), heads_per_group, a.stride(0), b.stride(0), out.stride(0), H, D, V, n_seg, unit_eps, D ** -0.5)
    c = None
    if chunks is not None:
        table, first, *ws = chunks
        n = table.shape[0]
        if any(t.numel() * t.element_size() < x for t, x in zip(ws, delta_workspace(n, H, H // heads_per_group, D, V))):
            raise ValueError("delta: workspace too small")
        c = DeltaChunks(_p(table), _p(first), *(_p(t) for t in ws), n, 0)
    _lib.check(_lib.load().dlp_layers_delta(C.byref(args), _ref(c), _ref(conv), 1 if c is not None else 2 if single else 0, api._stream()), "layers_delta")
    api._count(3 if c is not None else 1)
    return out


def delta_workspace(n_chunks: int, H: int, G: int, D: int, V: int) -> tuple[int, ...]:
    """Bytes of the workspaces of `delta` in chunks (G heads of queries and keys): states, keys, inverses, weights, writes, gates."""
    dp, vp, c = (64 if D <= 64 else 128), -(-V // 16) * 16, DELTA_CHUNK
    matrix = n_chunks * H * c * (c + 8) * 4
    return n_chunks * H * dp * vp * 4, n_chunks * G * c * (dp + 8) * 2, matrix, matrix, n_chunks * H * c * vp * 4, n_chunks * H * c * 20


def most_chunks(rows: int, size: int) -> int:
    """Chunks that a batch of this many rows can have at most: every long segment may end in a partial one."""
    return rows // size + rows // LONG_FROM + 1


def latent_tile_rows(H: int, T: int, Rc: int = 0) -> int:
    """(token, head) rows per tile: enough to fill the tensor-core rows, no more than a batch of single tokens has (nor, of wide rows Rc, than
    shared memory holds)."""
    bm = 64 if T * H > 4096 or H >= 48 else 32 if H > 16 else 16
    return bm if Rc <= 512 else min(bm, 32)


def latent_attention(q, cache, block_table, tok_slot, pos, tile_row0, tile_rows, n_tiles: int, bm: int, H: int, T: int, scale: float, out, n_splits: int = 1,
                     workspace=None, window: int = NO_WINDOW):
    """q [T, H * Rc] over the cached rows [..., Rc] of the last `window` tokens; their first Vc columns are the values, out [T, H * Vc]."""
    _need_cuda(cache, "latent_attention")
    po, pm = workspace if workspace is not None and n_splits > 1 else (None, None)
    a = LatentArgs(_p(q), _p(cache), _p(block_table), _p(tok_slot), _p(pos), _p(tile_row0), _p(tile_rows), _p(out), _p(po), _p(pm), block_table.shape[1],
                   cache.shape[-2], H, cache.shape[-1], out.shape[1] // H, T, n_tiles, bm, n_splits, window, scale)
    _lib.check(_lib.load().dlp_layers_latent_attention(C.byref(a), int(cache.dtype == torch.float32), api._stream()), "layers_latent_attention")
    api._count(2 if n_splits > 1 else 1)
    return out


def latent_gather(cache, block_table_row, S: int, out):
    """Latent rows 0 .. S-1 of one request out of its pages (from the row's first page on) -> out [S, Rc] (bf16)."""
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


def rows_attention(q, kv, S: int, pos0: int, H: int, Dp: int, Vp: int, V: int, scale: float, out, gate=None, window: int = NO_WINDOW):
    """Causal attention of q [T, H * Dp], rows pos0 .. of kv [S, H * (Dp + Vp)], to the last `window` rows; out [T, H * V], each head times sigmoid(gate)."""
    _need_cuda(q, "rows_attention")
    _lib.check(_lib.load().dlp_layers_rows_attention(_p(q), _p(kv), kv.stride(0), S, q.shape[0], pos0, H, Dp, Vp, V, window, scale, _p(gate),
                                                     gate.stride(0) if gate is not None else 0, _p(out), out.stride(0), api._stream()), "layers_rows_attention")
    api._count()
    return out


# ---- routed experts -------------------------------------------------------------------------------------------------------
def route(logits: torch.Tensor, rule: Routing, ids: torch.Tensor, weights: torch.Tensor, T: int):
    """Chosen experts and their weights -> ids, weights [T * top]."""
    _need_cuda(logits, "route")
    _lib.check(_lib.load().dlp_layers_route(_p(logits), logits.stride(0), C.byref(rule.c()), _p(ids), _p(weights), T, api._stream()), "layers_route")
    api._count()


def expert_matvec_fits(T: int, top: int, w: torch.Tensor, shared: torch.Tensor | None = None) -> bool:
    """The staged rows (one per token, or one per assignment in front of the down product) fit the shared memory of one block."""
    return T * (top * w.shape[1] + (shared.shape[1] if shared is not None else 0)) * w.element_size() <= 150 * 1024


def expert_matvec(st: RowStage, logits, rule: Routing, w: torch.Tensor, rows: int, out: torch.Tensor, T: int, down: bool, act: int = OUT_RELU2, shared=None) -> torch.Tensor:
    """1..4 staged rows times the matrices of their chosen experts, w [n * rows, ld]: activation -> out [T * top, ld] (activation type), or
    (down; st: one row per assignment) the weighted sum over a token's experts -> out [T, ld] fp32.  shared = (matrix, rows): an expert of every
    token, weighted by the sigmoid of logits column n; up: its output rows [T, ld], down: its input rows."""
    _need_cuda(w, "expert_matvec")
    a = ExpertArgs(_p(logits), rule.c(), _p(w), logits.stride(0), rows, w.stride(0), act)
    if shared is not None:
        m, r = shared
        a.w_s, a.rows_s, a.K_s, a.ldw_s = _p(m), m.shape[0], m.shape[1], m.stride(0)
        if down:
            a.x_s, a.ldx_s = _p(r), r.stride(0)
        else:
            a.act_s, a.ld_act_s = _p(r), r.stride(0)
    _lib.check(_lib.load().dlp_layers_expert_matvec(C.byref(st), C.byref(a), _p(out), out.stride(0), int(down), T, int(w.dtype == torch.float32), api._stream()),
               "layers_expert_matvec")
    api._count()
    return out


def expert_plan(ids: torch.Tensor, n_expert: int, tile: int, plan):
    """Expert-sorted order of the assignments and the row tiles of the grouped products (ops.api.MoePlan)."""
    _need_cuda(ids, "expert_plan")
    api.moe_plan(ids, n_expert, tile, plan)


def expert_gather(x: torch.Tensor, plan, top: int, n: int, out: torch.Tensor) -> torch.Tensor:
    """out[row] = x[token of the row]; rows are moved as 16-byte pieces, so fp32 rows count twice as many 2-byte elements."""
    _need_cuda(x, "expert_gather")
    api.moe_gather(x.view(torch.int16), plan, top, n, out.view(torch.int16))
    return out


def linear_grouped(xs: torch.Tensor, w: torch.Tensor, rows: int, n_expert: int, tile: int, plan, out: torch.Tensor, act: int = OUT_F32) -> torch.Tensor:
    """out[row] = xs[row] . W_e^T for every expert-sorted row (e: the row's expert; `rows` matrix rows each), one launch; OUT_RELU2, OUT_SWIGLU: in the
    activation type."""
    _need_cuda(xs, "linear_grouped")
    f32 = w.dtype == torch.float32
    ws = None if f32 else api.gemm_workspace(xs.device)
    _lib.check(_lib.load().dlp_layers_linear_grouped(_p(xs), xs.stride(0), _p(w), w.stride(0), rows, w.shape[1], _p(out), out.stride(0), act,
                                                     xs.shape[0], n_expert, tile, C.byref(plan.c), int(f32), _p(ws), 0 if ws is None else ws.numel(), api._stream()),
               "layers_linear_grouped")
    api._count()
    return out


def expert_combine(y: torch.Tensor, plan, weights: torch.Tensor, T: int, top: int, out: torch.Tensor, shared=None) -> torch.Tensor:
    """out[t] = sum of the weighted expert rows of token t, in the order of the choice; shared = (rows [T, E], gate logits [T, 1]): one more row each,
    weighted by the sigmoid of its logit."""
    ys, gs = shared if shared is not None else (None, None)
    _need_cuda(y, "expert_combine")
    _lib.check(_lib.load().dlp_layers_combine(_p(y), y.stride(0), _p(plan.pos), _p(weights), T, top, out.shape[1], _p(out), _p(ys), _p(gs), gs.stride(0) if gs is not None else 0, api._stream()), "layers_combine")
    api._count()
    return out


# ---- grouped-query attention (windows, chunks, one or two maps) ----------------------------------------------------------------------------------------
def gqa_tile(R: int, longest: int) -> tuple[int, int]:
    """Rows of a tile and the tokens it holds, for R query heads per key / value head and segments of up to `longest` tokens."""
    bm = 16 if longest * R <= 16 or longest == 1 else 64
    return bm, bm // min(R, bm)


def gqa_blocks(G: int, R: int, bm: int) -> int:
    """Blocks per tile and key range."""
    return G * -(-R // min(R, bm))


def gqa_args(shape, proj, kc, vc, block_table, tok_slot, pos, slot, out, T: int, q=None, tiles=None, bm: int = 16, n_splits: int = 1, mix=None) -> GqaArgs:
    """shape: models.mixers.Attention (heads, sizes, norms, rotation, window, chunk, maps); tiles: (first rows, rows, count) of the launch; mix: see
    `gqa_prepare`."""
    m = shape
    row0, rows, n = tiles if tiles is not None else (None, None, 0)
    return GqaArgs(_p(proj), _p(m.q_norm), _p(m.k_norm), _p(m.inv_freq), _p(q), _p(kc), _p(vc), _p(block_table), _p(tok_slot), _p(pos), _p(slot), _p(row0), _p(rows), _p(out),
                   proj.stride(0) if proj is not None else 0, out.stride(0) if out is not None else 0, T, m.H, m.G, m.D, m.V, m.Dc, m.Vc, m.rot, block_table.shape[1],
                   kc.shape[-2], kc.shape[0], n, bm, n_splits, m.window, m.keep, m.chunk, m.maps, int(m.adjacent), m.eps, m.scale, m.rot_scale,
                   *((_p(mix[0]), 1 if mix[1] is None else 2, mix[1] or 0.0) if mix is not None else (None, 0, 0.0)))


def gqa_prepare(m, proj, kc, vc, block_table, tok_slot, pos, slot, q, T: int, mix=None):
    """Projection rows -> normalised and rotated queries q [T, H * Dc]; keys and values into the pages.  mix = (values [T, G * V] fp32, share): this share
    of those values takes the place of the layer's own; share None: the layer's own values are kept there."""
    _need_cuda(kc, "gqa_prepare")
    a = gqa_args(m, proj, kc, vc, block_table, tok_slot, pos, slot, None, T, q=q, mix=mix)
    _lib.check(_lib.load().dlp_layers_gqa_prepare(C.byref(a), int(kc.dtype == torch.float32), api._stream()), "layers_gqa_prepare")
    api._count()


def gqa_attention(m, q, kc, vc, block_table, tok_slot, pos, tiles, bm: int, n_splits: int, out, T: int):
    """Prepared queries over the cached keys their window shows, tiles of up to bm (token, head) rows of one key / value head."""
    _need_cuda(kc, "gqa_attention")
    a = gqa_args(m, None, kc, vc, block_table, tok_slot, pos, None, out, T, q=q, tiles=tiles, bm=bm, n_splits=n_splits)
    _lib.check(_lib.load().dlp_layers_gqa_attention(C.byref(a), 0, int(kc.dtype == torch.float32), api._stream()), "layers_gqa_attention")
    api._count()
    return out


def gqa_decode(m, proj, kc, vc, block_table, tok_slot, pos, tiles, n_splits: int, out, T: int, mix=None):
    """Single tokens straight from the projection: norm, rotation, cache write and attention in one launch (bf16)."""
    _need_cuda(kc, "gqa_decode")
    a = gqa_args(m, proj, kc, vc, block_table, tok_slot, pos, None, out, T, tiles=tiles, n_splits=n_splits, mix=mix)
    _lib.check(_lib.load().dlp_layers_gqa_attention(C.byref(a), 1, 0, api._stream()), "layers_gqa_attention")
    api._count()
    return out


def gqa_flash(m, q, kc, vc, block_table, tok_slot, pos, tiles, out, T: int):
    """Prepared queries in tiles of 128 consecutive tokens (tcgen05 flash kernel, bf16)."""
    _need_cuda(kc, "gqa_flash")
    a = gqa_args(m, None, kc, vc, block_table, tok_slot, pos, None, out, T, q=q, tiles=tiles)
    _lib.check(_lib.load().dlp_layers_gqa_flash(C.byref(a), api._stream()), "layers_gqa_flash")
    api._count()
    return out


def check_waits():
    """Raise if a wait inside an attention kernel gave up since the last call (synchronises the device)."""
    flag = C.c_int(0)
    _lib.check(_lib.load().dlp_layers_rows_attention_error(C.byref(flag)), "rows_attention_error")
    if flag.value:
        raise _lib.DlpError("a wait inside the attention kernel ran into its limit")
