"""Model folders: config.json + model.safetensors, and the registry of architectures they may name.

A folder's `architecture` selects a reader below, which turns config.json into a ModelConfig with a layer list.  GGUF files keep their
own reader (gguf/, models/config.py); `open_model` takes either.
"""
from __future__ import annotations

import json
import mmap
import os
import struct
from dataclasses import dataclass

import torch

from .config import LayerSpec, ModelConfig

_ST_TYPES = {"BF16": torch.bfloat16, "F16": torch.float16, "F32": torch.float32, "F64": torch.float64, "I32": torch.int32, "I64": torch.int64,
             "I16": torch.int16, "I8": torch.int8, "U8": torch.uint8, "BOOL": torch.bool}


class SafetensorsFile:
    """Memory-mapped safetensors file: u64 header length, JSON header (name -> dtype, shape, data_offsets), tensor bytes."""

    def __init__(self, path: str):
        self.path = path
        with open(path, "rb") as f:
            size = os.fstat(f.fileno()).st_size
            if size < 8:
                raise ValueError(f"{path}: not a safetensors file")
            n = struct.unpack("<Q", f.read(8))[0]
            if n > size - 8:
                raise ValueError(f"{path}: header of {n} bytes in a file of {size}")
            head = json.loads(f.read(n))
            self._map = mmap.mmap(f.fileno(), 0, access=mmap.ACCESS_READ)
        self.metadata = head.pop("__metadata__", {})
        self.entries = head
        self._base = 8 + n
        for name, e in head.items():
            lo, hi = e["data_offsets"]
            if e["dtype"] not in _ST_TYPES:
                raise ValueError(f"{path}: {name} has the unknown type {e['dtype']}")
            want = _ST_TYPES[e["dtype"]].itemsize
            for d in e["shape"]:
                want *= d
            if lo < 0 or hi - lo != want or self._base + hi > size:
                raise ValueError(f"{path}: {name} does not fit its bytes")

    def __contains__(self, name: str) -> bool:
        return name in self.entries

    def tensor(self, name: str) -> torch.Tensor:
        """A copy of the tensor on the host."""
        if name not in self.entries:
            raise KeyError(f"{self.path}: no tensor {name!r}")
        e = self.entries[name]
        lo, hi = e["data_offsets"]
        raw = bytearray(self._map[self._base + lo:self._base + hi])
        dt = _ST_TYPES[e["dtype"]]
        return torch.frombuffer(raw, dtype=dt).view(e["shape"]) if raw else torch.empty(e["shape"], dtype=dt)

    def nbytes(self) -> int:
        return sum(e["data_offsets"][1] - e["data_offsets"][0] for e in self.entries.values())


def write_safetensors(path: str, tensors: dict[str, torch.Tensor]) -> str:
    names = {v: k for k, v in _ST_TYPES.items()}
    head, off = {}, 0
    for n, t in tensors.items():
        nb = t.numel() * t.element_size()
        head[n] = {"dtype": names[t.dtype], "shape": list(t.shape), "data_offsets": [off, off + nb]}
        off += nb
    hj = json.dumps(head).encode()
    hj += b" " * (-len(hj) % 8)
    with open(path, "wb") as f:
        f.write(struct.pack("<Q", len(hj)) + hj)
        for t in tensors.values():
            if t.numel():
                f.write(t.detach().cpu().contiguous().view(-1).view(torch.uint8).numpy().tobytes())
    return path


# ---- architectures -------------------------------------------------------------------------------------------------
def _need(what: str, d, keys: tuple[str, ...]):
    """Check that `d` has these keys, dotted ones inside nested objects: positive sizes, except where a rule below says otherwise."""
    rules = {"scale": lambda v: isinstance(v, (int, float)), "base": lambda v: isinstance(v, (int, float)) and v > 0,
             "keep_first": lambda v: isinstance(v, int) and v >= 0}
    for path in keys:
        v = d
        for k in path.split("."):
            if not isinstance(v, dict) or k not in v:
                raise ValueError(f"{what}: {path} missing")
            v = v[k]
        if not rules.get(k, lambda v: isinstance(v, int) and v >= 1)(v):
            raise ValueError(f"{what}: {path} = {v!r}")


def _layer_list(cfg: dict, mixers: dict[str, tuple[str, ...]], mlps: dict[str, tuple[str, ...]]) -> tuple[LayerSpec, ...]:
    """Check every entry's type and sizes: `mixers` / `mlps` name the keys each kind must have."""
    out = []
    for i, e in enumerate(cfg["layers"]):
        if e["type"] not in mixers:
            raise ValueError(f"layer {i}: unknown mixer {e['type']!r}")
        _need(f"layer {i} ({e['type']})", e["mixer"], mixers[e["type"]])
        mlp = e.get("mlp")
        if mlp is not None:
            if mlp.get("kind") not in mlps:
                raise ValueError(f"layer {i}: unknown feed-forward {mlp.get('kind')!r}")
            _need(f"layer {i} (feed-forward)", mlp, mlps[mlp["kind"]])
        out.append(LayerSpec(e["type"], dict(e["mixer"]), dict(mlp) if mlp is not None else None))
    return tuple(out)


def _layered_config(name: str, cfg: dict, layers: tuple[LayerSpec, ...], **kw) -> ModelConfig:
    return ModelConfig(name=name, arch=name, vocab_size=cfg["vocab"], n_embd=cfg["width"], n_layer=len(layers), n_head=0, n_head_kv=0, head_dim=0, n_ff=0,
                       n_ctx_train=int(cfg.get("context", 1 << 20)), rms_eps=float(cfg["norm"]["eps"]), rope_dim=0, bos_id=-1, eos_id=-1, layers=layers, **kw)


def talizen_config(cfg: dict) -> ModelConfig:
    """Talizen: HGRN2 and latent-attention layers in any order, tanh-gelu gated feed-forward or none, grouped norms behind the sublayers."""
    layers = _layer_list(cfg, {"hgrn2": ("heads", "dim", "vdim"), "latent_attention": ("heads", "dim", "vdim", "kv_rank", "scale")}, {"dense": ("ff",)})
    groups = cfg["norm"]["groups"]
    if cfg["width"] % groups:
        raise ValueError(f"{groups} norm groups do not divide the width {cfg['width']}")
    return _layered_config("talizen", cfg, layers, norm_groups=groups, pre_norm=False, post_norm=True)


def vozinex_config(cfg: dict) -> ModelConfig:
    """Vozinex: windowed grouped-query attention with kept first tokens, routed experts or no feed-forward, layer norms in front of the
    sublayers, a range of layers that runs several times."""
    layers = _layer_list(cfg, {"attention": ("heads", "kv_heads", "dim", "vdim", "rot.dims", "rot.base", "scale", "mask.size", "mask.keep_first")},
                         {"moe": ("expert.ff", "router.experts", "router.top")})
    for i, s in enumerate(layers):
        m = s.mixer
        if m["heads"] % m["kv_heads"]:
            raise ValueError(f"layer {i}: {m['kv_heads']} key / value heads do not divide {m['heads']} heads")
        if m["rot"]["dims"] % 2 or m["rot"]["dims"] > m["dim"]:
            raise ValueError(f"layer {i}: rotation of {m['rot']['dims']} of {m['dim']} dimensions")
        if s.mlp and s.mlp["router"]["top"] > s.mlp["router"]["experts"]:
            raise ValueError(f"layer {i}: {s.mlp['router']['top']} of {s.mlp['router']['experts']} experts")
    loop = ()
    if cfg.get("loop"):
        loop = tuple(cfg["loop"].get(k) for k in ("start", "stop", "times"))
        if not (all(isinstance(x, int) for x in loop) and 0 <= loop[0] < loop[1] <= len(layers) and loop[2] >= 1):
            raise ValueError(f"loop {cfg['loop']!r} does not fit {len(layers)} layers")
    return _layered_config("vozinex", cfg, layers, norm_type="layer", loop=loop)


ARCHITECTURES = {"Talizen": talizen_config, "Vozinex": vozinex_config}


@dataclass
class ModelDir:
    path: str
    config: dict
    cfg: ModelConfig
    tensors: SafetensorsFile

    @property
    def metadata(self) -> dict:
        """Tokenizer-free stand-in for a GGUF file's metadata (the vocabulary is the token numbers: utils/tokenizer.py `IdTokenizer`)."""
        return {"general.name": os.path.basename(os.path.abspath(self.path)), "general.architecture": self.cfg.arch}


def is_model_dir(path) -> bool:
    return isinstance(path, (str, os.PathLike)) and os.path.isfile(os.path.join(path, "config.json"))


def open_model_dir(path: str) -> ModelDir:
    with open(os.path.join(path, "config.json")) as f:
        config = json.load(f)
    arch = config.get("architecture")
    if arch not in ARCHITECTURES:
        raise ValueError(f"{path}: unknown architecture {arch!r} (known: {', '.join(sorted(ARCHITECTURES))})")
    return ModelDir(path, config, ARCHITECTURES[arch](config), SafetensorsFile(os.path.join(path, "model.safetensors")))


def open_model(path: str):
    """A model folder or a GGUF file."""
    if is_model_dir(path):
        return open_model_dir(path)
    from ..gguf import open_gguf
    return open_gguf(path)


def make_engine(weights, **kw):
    """The engine class of a loaded model."""
    if weights.cfg.layers:
        from .layered import LayeredEngine
        return LayeredEngine(weights, **kw)
    from .llama import LlamaEngine
    return LlamaEngine(weights, **kw)
