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
    number = lambda v: isinstance(v, (int, float)) and not isinstance(v, bool)
    positive = lambda v: number(v) and v > 0
    rules = {"scale": number, "diff": number, "base": positive, "factor": positive, "low": positive, "high": positive, "original": positive, "fast": positive, "slow": positive,
             "logit_scale": number, "keep_first": lambda v: isinstance(v, int) and v >= 0, "decay": lambda v: isinstance(v, list) and all(number(x) and 0 <= x <= 1 for x in v)}
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
    for s in layers:
        if s.type == "latent_attention":
            s.mixer["gate"] = True
    groups = cfg["norm"]["groups"]
    if cfg["width"] % groups:
        raise ValueError(f"{groups} norm groups do not divide the width {cfg['width']}")
    return _layered_config("talizen", cfg, layers, norm_groups=groups, pre_norm=False, post_norm=True)


def _loop(cfg: dict, layers) -> tuple:
    if not cfg.get("loop"):
        return ()
    loop = tuple(cfg["loop"].get(k) for k in ("start", "stop", "times"))
    if not (all(isinstance(x, int) for x in loop) and 0 <= loop[0] < loop[1] <= len(layers) and loop[2] >= 1):
        raise ValueError(f"loop {cfg['loop']!r} does not fit {len(layers)} layers")
    return loop


def _check_attention(what: str, m: dict):
    if m["heads"] % m["kv_heads"]:
        raise ValueError(f"{what}: {m['kv_heads']} key / value heads do not divide {m['heads']} heads")
    if m["rot"]["dims"] % 2 or m["rot"]["dims"] > m["dim"]:
        raise ValueError(f"{what}: rotation of {m['rot']['dims']} of {m['dim']} dimensions")


def vozinex_config(cfg: dict) -> ModelConfig:
    """Vozinex: windowed grouped-query attention with kept first tokens, routed experts or no feed-forward, layer norms in front of the
    sublayers, a range of layers that runs several times."""
    layers = _layer_list(cfg, {"attention": ("heads", "kv_heads", "dim", "vdim", "rot.dims", "rot.base", "scale", "mask.size", "mask.keep_first")},
                         {"moe": ("expert.ff", "router.experts", "router.top")})
    for i, s in enumerate(layers):
        _check_attention(f"layer {i}", s.mixer)
        s.mixer["qk_norm"] = True
        if s.mlp and s.mlp["router"]["top"] > s.mlp["router"]["experts"]:
            raise ValueError(f"layer {i}: {s.mlp['router']['top']} of {s.mlp['router']['experts']} experts")
    return _layered_config("vozinex", cfg, layers, norm_type="layer", loop=_loop(cfg, layers), loop_rejoin=True)


def nifalorn_config(cfg: dict) -> ModelConfig:
    """Nifalorn: lightning attention, Mamba-2 and chunked differential attention in any order; dense squared-ReLU feed-forward, routed experts
    with a shared one, or none; RMS norms with weights around zero in front of the sublayers; a range of layers that runs several times."""
    layers = _layer_list(cfg, {"lightning": ("heads", "dim", "vdim", "decay"), "mamba2": ("heads", "vdim", "state", "groups", "conv", "norm_groups"),
                               "attention": ("heads", "kv_heads", "dim", "vdim", "rot.dims", "rot.base", "scale", "mask.size", "diff")},
                         {"dense": ("ff",), "moe": ("expert.ff", "router.experts", "router.top")})
    out = []
    for i, s in enumerate(layers):
        m, mlp, what = dict(s.mixer), s.mlp, f"layer {i}"
        if s.type == "lightning" and len(m["decay"]) != m["heads"]:
            raise ValueError(f"{what}: {len(m['decay'])} decays for {m['heads']} heads")
        if s.type == "mamba2":
            if m["heads"] % m["groups"] or m["heads"] * m["vdim"] % m["norm_groups"]:
                raise ValueError(f"{what}: {m['groups']} groups, {m['norm_groups']} norm groups of {m['heads']} heads of {m['vdim']}")
            if m["conv"] > 32:
                raise ValueError(f"{what}: a convolution over {m['conv']} tokens (at most 32)")
        if s.type == "attention":
            _check_attention(what, m)
            scaling = m["rot"].get("scaling")
            if scaling is not None:
                _need(what, scaling, ("factor", "low", "high", "original"))
                if scaling["low"] >= scaling["high"]:
                    raise ValueError(f"{what}: rotation scaling {scaling!r}")
            m["rot"], m["mask"] = {**m["rot"], "adjacent": True}, {"chunk": m["mask"]["size"]}
        if mlp is not None and mlp["kind"] == "dense":
            mlp = {**mlp, "kind": "relu2"}
        elif mlp is not None:
            r = {"groups": {"count": 1, "keep": 1}, "scale": 1.0, **{k: v for k, v in mlp["router"].items() if v is not None}}
            _need(what, r, ("scale", "groups.count", "groups.keep"))
            if mlp.get("shared"):
                _need(what, mlp, ("shared.ff",))
            n, count, keep = r["experts"], r["groups"]["count"], r["groups"]["keep"]
            if n % count or keep > count or r["top"] > keep * (n // count):
                raise ValueError(f"{what}: {r['top']} of {n} experts in {keep} of {count} groups")
            mlp = {**mlp, "expert": {**mlp["expert"], "gated": True}, "router": {**r, "score": "sigmoid"}}
        out.append(LayerSpec(s.type, m, mlp))
    cfg = {"embedding": {"scale": 1.0}, "logit_scale": 1.0, **cfg}
    _need("config", cfg, ("embedding.scale", "logit_scale"))
    if not cfg["logit_scale"]:
        raise ValueError("logit_scale = 0")
    return _layered_config("nifalorn", cfg, tuple(out), loop=_loop(cfg, layers), norm_offset=1.0, embedding_scale=float(cfg["embedding"]["scale"]),
                           logit_scale=1.0 / float(cfg["logit_scale"]))


def rigalorn_config(cfg: dict) -> ModelConfig:
    """Rigalorn: windowed attention with biases, YaRN rotation and values mixed across layers, the gated delta rule, and latent attention with
    low-rank queries and a windowed rotated part, in any order; mixer and xIELU feed-forward (or none) side by side behind one RMS norm."""
    layers = _layer_list(cfg, {"attention": ("heads", "kv_heads", "dim", "vdim", "rot.dims", "rot.base", "scale"), "delta": ("heads", "kv_heads", "dim", "vdim", "conv"),
                               "latent_attention": ("heads", "dim", "vdim", "q_rank", "kv_rank", "rot_dim", "rot.dims", "rot.base", "scale")}, {"dense": ("ff",)})
    out, values = [], None
    for i, s in enumerate(layers):
        m, what = dict(s.mixer), f"layer {i}"
        if s.type == "delta":
            if m["heads"] % m["kv_heads"]:
                raise ValueError(f"{what}: {m['kv_heads']} query / key heads do not divide {m['heads']} heads")
            if m["conv"] > 32:
                raise ValueError(f"{what}: a convolution over {m['conv']} tokens (at most 32)")
        else:
            if m.get("mask"):
                _need(what, m, ("mask.size",))
            scaling = m["rot"].get("scaling")
            if scaling is not None:
                _need(what, scaling, ("factor", "fast", "slow", "original"))
                if m["rot"]["base"] == 1:
                    raise ValueError(f"{what}: scaled rotation of base 1")
        if s.type == "attention":
            _check_attention(what, m)
            m["bias"] = True
            if m.get("v_mix"):
                size = m["kv_heads"], m["vdim"]
                if values not in (None, size):
                    raise ValueError(f"{what}: mixes values of {values[0]} heads of {values[1]} into {size[0]} of {size[1]}")
                m["v_mix"], values = "first" if values is None else "later", size
        if s.type == "latent_attention" and (m["rot"]["dims"] != m["rot_dim"] or m["rot_dim"] % 2):
            raise ValueError(f"{what}: rotation of {m['rot']['dims']} of {m['rot_dim']} dimensions")
        out.append(LayerSpec(s.type, m, {**s.mlp, "kind": "xielu"} if s.mlp is not None else None))
    cfg = {"embedding": {"scale": 1.0}, **cfg}
    _need("config", cfg, ("embedding.scale",))
    return _layered_config("rigalorn", cfg, tuple(out), embedding_scale=float(cfg["embedding"]["scale"]), parallel_residual=True)


ARCHITECTURES = {"Talizen": talizen_config, "Vozinex": vozinex_config, "Nifalorn": nifalorn_config, "Rigalorn": rigalorn_config}


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
