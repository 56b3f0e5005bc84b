"""Small random layer-list models for the tests, and a way to run the engine's bookkeeping without a GPU."""
from __future__ import annotations

import itertools
import json
import os

import torch

import plain_layers as plain
from distributed_llm_pipeline_b200.models.modeldir import write_safetensors


def hgrn2(heads, dim, vdim, ff=None):
    return {"type": "hgrn2", "mixer": {"heads": heads, "dim": dim, "vdim": vdim}, "mlp": None if ff is None else {"kind": "dense", "ff": ff}}


def latent(heads, dim, vdim, rank, scale, ff=None):
    return {"type": "latent_attention", "mixer": {"heads": heads, "dim": dim, "vdim": vdim, "kv_rank": rank, "scale": scale},
            "mlp": None if ff is None else {"kind": "dense", "ff": ff}}


def attention(heads, kv_heads, dim, vdim, scale, rot, size, keep, experts=None, top=None, ff=None, base=10000.0):
    return {"type": "attention", "mixer": {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "scale": scale, "rot": {"dims": rot, "base": base},
                                           "mask": {"size": size, "keep_first": keep}},
            "mlp": None if experts is None else {"kind": "moe", "expert": {"ff": ff}, "router": {"experts": experts, "top": top}}}


def lightning(heads, dim, vdim, decay=None, mlp=None):
    return {"type": "lightning", "mixer": {"heads": heads, "dim": dim, "vdim": vdim, "decay": decay or [1 - 2.0 ** (-1 - 2 * i) for i in range(heads)]}, "mlp": mlp}


def mamba2(heads, vdim, state, groups, conv, norm_groups, mlp=None):
    return {"type": "mamba2", "mixer": {"heads": heads, "vdim": vdim, "state": state, "groups": groups, "conv": conv, "norm_groups": norm_groups}, "mlp": mlp}


def differential(heads, kv_heads, dim, vdim, scale, rot, size, diff, mlp=None, base=10000.0, scaling=(4.0, 1.0, 4.0, 64)):
    return {"type": "attention", "mixer": {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "scale": scale, "diff": diff, "mask": {"size": size},
                                           "rot": {"dims": rot, "base": base, "scaling": dict(zip(("factor", "low", "high", "original"), scaling))}}, "mlp": mlp}


def delta(heads, kv_heads, dim, vdim, conv, ff=None):
    return {"type": "delta", "mixer": {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "conv": conv}, "mlp": None if ff is None else dense(ff)}


def biased_attention(heads, kv_heads, dim, vdim, scale, rot, size, v_mix=True, ff=None, base=10000.0, yarn=(8.0, 64, 32.0, 1.0)):
    r = {"dims": rot, "base": base, **({"scaling": dict(zip(("factor", "original", "fast", "slow"), yarn))} if yarn else {})}
    return {"type": "attention", "mixer": {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "scale": scale, "rot": r, "mask": {"size": size}, "v_mix": v_mix},
            "mlp": None if ff is None else dense(ff)}


def low_rank_latent(heads, dim, rot, vdim, q_rank, rank, scale, size, ff=None, base=10000.0):
    return {"type": "latent_attention", "mixer": {"heads": heads, "dim": dim, "rot_dim": rot, "vdim": vdim, "q_rank": q_rank, "kv_rank": rank, "scale": scale, "mask": {"size": size},
                                                  "rot": {"dims": rot, "base": base}}, "mlp": None if ff is None else dense(ff)}


def rigalorn(width, vocab, layers, eps=1e-5, emb=1.0):
    return {"architecture": "Rigalorn", "width": width, "vocab": vocab, "norm": {"eps": eps}, "layers": layers, "embedding": {"scale": emb}}


def dense(ff):
    return {"kind": "dense", "ff": ff}


def shared_moe(experts, top, ff, shared, count=1, keep=1, scale=1.0):
    return {"kind": "moe", "expert": {"ff": ff}, "router": {"experts": experts, "top": top, "groups": {"count": count, "keep": keep}, "scale": scale}, "shared": {"ff": shared}}


def nifalorn(width, vocab, layers, loop=None, eps=1e-5, emb=1.0, logit=1.0):
    start, stop, times = loop or (0, len(layers), 1)
    return {"architecture": "Nifalorn", "width": width, "vocab": vocab, "norm": {"eps": eps}, "layers": layers, "loop": {"start": start, "stop": stop, "times": times},
            "embedding": {"scale": emb}, "logit_scale": logit}


def vozinex(width, vocab, layers, loop=None, eps=1e-5):
    start, stop, times = loop or (0, len(layers), 1)
    return {"architecture": "Vozinex", "width": width, "vocab": vocab, "norm": {"eps": eps}, "layers": layers, "loop": {"start": start, "stop": stop, "times": times}}


def config(width, vocab, groups, layers, eps=1e-5):
    return {"architecture": "Talizen", "width": width, "vocab": vocab, "norm": {"groups": groups, "eps": eps}, "layers": layers}


CONFIGS = {
    # sizes that are no multiple of a vector load, an odd vocabulary, both mixers with and without a feed-forward
    "odd": config(72, 101, 3, [latent(5, 12, 20, 40, 0.31, 52), hgrn2(3, 20, 12, 36), hgrn2(1, 36, 28), latent(2, 44, 8, 24, 0.2)], eps=3e-4),
    # one group, one head
    "single": config(64, 48, 1, [hgrn2(1, 64, 64), latent(1, 64, 64, 32, 1.0, 64), hgrn2(2, 32, 32, 96)]),
    # wide heads: 128-channel states, a latent above 128 columns, more heads than one 16-row tile
    "wide": config(256, 320, 4, [hgrn2(2, 128, 128, 256), latent(20, 32, 32, 160, 0.15, 192), hgrn2(2, 160, 48)]),
    # channels beyond every register-resident size but the last, latent beyond the tensor-core form
    "huge": config(64, 80, 2, [hgrn2(1, 300, 20), latent(3, 40, 24, 544, 0.1), hgrn2(1, 8, 8)]),
    "recurrent": config(48, 60, 2, [hgrn2(2, 24, 24), hgrn2(2, 16, 40, 80)]),
    # windowed attention and experts: partial rotation, value size unlike key size, sizes that are no multiple of a vector load, windows of
    # different size, a loop in the middle that runs twice
    "experts": vozinex(72, 101, [attention(6, 2, 20, 12, 0.4, 12, 24, 5, 7, 2, 20), attention(4, 4, 16, 24, 0.3, 16, 33, 0), attention(6, 1, 24, 20, 0.35, 8, 17, 9, 5, 3, 36),
                                 attention(3, 3, 12, 12, 0.5, 2, 1000, 3, 4, 4, 8, base=500.0)], loop=(1, 3, 2), eps=3e-4),
    # one layer, looped from the start to the end; one expert of one
    "loop": vozinex(64, 48, [attention(4, 1, 32, 32, 0.3, 32, 40, 4, 1, 1, 40)], loop=(0, 1, 3)),
    # heads of 128 and 64 (flash kernel), more query heads per key / value head than a 16-row tile, many experts
    "grouped": vozinex(256, 320, [attention(8, 2, 128, 64, 0.12, 64, 150, 20, 40, 6, 64), attention(20, 1, 64, 128, 0.15, 64, 64, 64, 9, 1, 72),
                                  attention(8, 4, 48, 80, 0.2, 48, 200, 1)], loop=(0, 2, 2)),
    # heads wider than the tensor-core forms take, next to a mask that shows one key
    "broad": vozinex(96, 64, [attention(2, 1, 264, 40, 0.1, 100, 50, 2, 3, 2, 24), attention(2, 2, 160, 192, 0.1, 160, 70, 3), attention(4, 2, 8, 8, 0.5, 8, 1, 1)]),
    # every mixer and feed-forward of Nifalorn at sizes that are no multiple of a vector load; a loop in the middle; scales unlike 1
    "hybrid": nifalorn(72, 101, [lightning(3, 20, 12, mlp=dense(52)), mamba2(4, 12, 20, 2, 4, 3, mlp=shared_moe(8, 2, 20, 28, 4, 2, 1.7)),
                                 differential(6, 2, 20, 12, 0.4, 12, 24, 0.35, mlp=shared_moe(12, 3, 36, 12, 3, 2, 0.6)), lightning(5, 8, 24)], loop=(1, 3, 2), eps=3e-4, emb=3.0, logit=0.5),
    # recurrences only: heads that keep everything or nothing, convolutions over one, two and six tokens, columns that are no multiple of four, one
    # group or one per head, one norm group or one per head
    "scalar": nifalorn(48, 60, [lightning(3, 16, 10, decay=[0.0, 1.0, 0.5], mlp=dense(20)), mamba2(3, 10, 7, 3, 1, 1), mamba2(4, 16, 24, 1, 6, 4, mlp=dense(64)), mamba2(6, 8, 16, 2, 2, 6)],
                       loop=(0, 2, 2), logit=3.0),
    # two maps per head: heads for the flash kernel, more query rows per key / value head than a tile, keys beyond the tensor-core forms; chunks
    # below and above a page, one token, more than the sequence
    "maps": nifalorn(128, 320, [differential(4, 2, 64, 128, 0.12, 64, 150, 0.6, mlp=shared_moe(40, 6, 64, 72, 8, 3, 2.5)), differential(20, 1, 24, 40, 0.2, 8, 70, 0.2),
                                differential(2, 2, 136, 24, 0.1, 100, 33, 0.8, scaling=(8.0, 1.0, 4.0, 2048)), differential(3, 3, 12, 20, 0.4, 2, 1, -0.3, mlp=shared_moe(3, 3, 8, 16)),
                                differential(2, 1, 96, 64, 0.1, 96, 1000, 0.0)], loop=(0, 1, 2), emb=11.0),
    # states of every register-resident size and beyond
    "states": nifalorn(96, 64, [lightning(2, 128, 128, mlp=dense(96)), lightning(1, 160, 72), mamba2(2, 64, 256, 1, 4, 2), mamba2(2, 20, 300, 2, 3, 1), mamba2(4, 32, 128, 2, 4, 1)], emb=0.5),
    # every mixer of Rigalorn, with and without a feed-forward, at sizes that are no multiple of a vector load; windows below a page; the first layer
    # that mixes values is not the first attention
    "parallel": rigalorn(72, 101, [biased_attention(6, 2, 20, 12, 0.4, 12, 24, v_mix=False, ff=52), low_rank_latent(5, 12, 6, 20, 28, 40, 0.35, 19, ff=36), delta(6, 2, 20, 12, 3, ff=52),
                                   biased_attention(4, 2, 16, 24, 0.3, 16, 9, yarn=None), delta(3, 3, 12, 10, 1), biased_attention(2, 2, 24, 24, 0.35, 8, 33, ff=20, base=500.0),
                                   low_rank_latent(3, 8, 2, 12, 17, 25, 0.5, 40)], eps=3e-4, emb=3.0),
    # delta rules only: one head, one group, long and short convolutions, states of every register-resident size and beyond
    "deltas": rigalorn(64, 60, [delta(4, 1, 64, 48, 4, ff=40), delta(2, 2, 128, 128, 2, ff=64), delta(1, 1, 160, 40, 6), delta(2, 1, 300, 12, 3), delta(5, 5, 8, 7, 32, ff=24)], eps=1e-3),
    # heads and latents for every form of the attentions: expanded keys of 64, 128 and 192, beyond them, latents above 512, more heads than a tile;
    # windows above a page and a key tile, one token, more than the sequence
    "windows": rigalorn(256, 320, [low_rank_latent(4, 48, 16, 64, 96, 96, 0.14, 70, ff=96), biased_attention(8, 2, 128, 64, 0.12, 64, 150, ff=128, yarn=(4.0, 40, 8.0, 0.5)),
                                   low_rank_latent(2, 128, 64, 128, 160, 512, 0.1, 131, ff=72), biased_attention(6, 2, 64, 64, 0.15, 64, 1), low_rank_latent(20, 40, 24, 24, 64, 160, 0.15, 1000),
                                   low_rank_latent(1, 200, 8, 40, 32, 544, 0.1, 33, ff=8)], emb=11.0),
    "attention": config(80, 64, 5, [latent(4, 16, 24, 32, 0.4, 40), latent(49, 8, 4, 64, 0.4)]),
}


CODE = 8     # models with routed experts: leading dimensions that only the embedding writes and only the routers read, as signs, so that no routing is a close call
             # (a model in bf16 would choose other experts there, and the comparison with exact arithmetic would say nothing)


def nifalorn_weights(cfg: dict, g, rnd, mat) -> dict[str, torch.Tensor]:
    E, V = cfg["width"], cfg["vocab"]
    w = {"embed": rnd(V, E, scale=1 / cfg["embedding"]["scale"]), "head": mat(V, E, 2.0 / cfg["logit_scale"]), "final.norm": rnd(E, scale=0.2)}
    w["embed"][:, :CODE] = (torch.randint(0, 2, (V, CODE), generator=g) * 8 - 4).to(torch.bfloat16) / cfg["embedding"]["scale"]
    for i, s in enumerate(cfg["layers"]):
        p, m, mix = f"l{i}.", s["mixer"], f"l{i}.mix."
        w[p + "norm1"] = rnd(E, scale=0.2)
        H, Vd = m["heads"], m["vdim"]
        if s["type"] == "lightning":
            D = m["dim"]
            w.update({mix + "q": mat(H * D, E, 1.5), mix + "k": mat(H * D, E, 1.5), mix + "v": mat(H * Vd, E, 1.5), mix + "g": mat(H * Vd, E, 1.5), mix + "norm": rnd(H * Vd, scale=0.2, mean=1.0)})
        elif s["type"] == "mamba2":
            ch = H * Vd + 2 * m["groups"] * m["state"]
            w.update({mix + "in": mat(H * Vd + ch + H, E, 1.5), mix + "conv": rnd(ch, m["conv"], scale=m["conv"] ** -0.5), mix + "conv.b": rnd(ch, scale=0.3),
                      mix + "dt_bias": rnd(H, scale=1.5, mean=-1.5), mix + "A_log": rnd(H, scale=1.0), mix + "D": rnd(H, mean=1.0, scale=0.5), mix + "norm": rnd(H * Vd, scale=0.2, mean=1.0)})
        else:
            G, D = m["kv_heads"], m["dim"]
            sharp = (2.5 / (m["scale"] * D ** 0.5)) ** 0.5          # scores of a few units, so that single keys count
            w.update({mix + "q": mat(2 * H * D, E, sharp), mix + "k": mat(2 * G * D, E, sharp), mix + "v": mat(G * Vd, E, 1.5)})
            w.update({mix + n: rnd(D, scale=0.3 * D ** -0.25) for n in ("lq1", "lk1", "lq2", "lk2")})
        w[mix + "o"] = mat(E, H * Vd)
        w[mix + "o"][:CODE] = 0
        if s["mlp"] is None:
            continue
        w[p + "norm2"] = rnd(E, scale=0.2)
        w[p + "norm2"][:CODE] = 0
        if s["mlp"]["kind"] == "dense":
            w.update({p + "mlp.up": mat(s["mlp"]["ff"], E), p + "mlp.down": mat(E, s["mlp"]["ff"])})
            w[p + "mlp.down"][:CODE] = 0
            continue
        n, ff = s["mlp"]["router"]["experts"], s["mlp"]["expert"]["ff"]
        for name, f in [(f"e{e}", ff) for e in range(n)] + [("shared", s["mlp"]["shared"]["ff"])]:
            w.update({p + f"mlp.{name}.gate": mat(f, E, 1.5), p + f"mlp.{name}.up": mat(f, E), p + f"mlp.{name}.down": mat(E, f)})
            w[p + f"mlp.{name}.down"][:CODE] = 0
        signs = torch.tensor(list(itertools.combinations(range(CODE), CODE // 2)))
        r = torch.zeros(n, E)
        r[:, :CODE] = -0.15
        r.scatter_(1, signs[torch.randperm(len(signs), generator=g)[:n]], 0.15)
        w.update({p + "mlp.router": r.to(torch.bfloat16), p + "mlp.correction": (-0.04 * ((torch.randperm(n, generator=g) + 1) / n) ** 1.3).to(torch.bfloat16), p + "mlp.shared.sg": mat(1, E, 1.5)})
    return w


def rigalorn_weights(cfg: dict, g, rnd, mat) -> dict[str, torch.Tensor]:
    E, V = cfg["width"], cfg["vocab"]
    w = {"embed": rnd(V, E, scale=1 / cfg["embedding"]["scale"]), "head": mat(V, E, 2.0), "final.norm": rnd(E, scale=0.2, mean=1.0)}
    for i, s in enumerate(cfg["layers"]):
        p, m, mix = f"l{i}.", s["mixer"], f"l{i}.mix."
        w[p + "norm1"] = rnd(E, scale=0.2, mean=1.0)
        H, D, Vd = m["heads"], m["dim"], m["vdim"]
        if s["type"] == "delta":
            G, taps = m["kv_heads"], m["conv"]
            for n, rows in (("q", G * D), ("k", G * D), ("v", H * Vd)):
                w.update({mix + n: mat(rows, E, 1.5), mix + n + ".conv": rnd(rows, taps, scale=taps ** -0.5, mean=0.3)})
            w.update({mix + "g": mat(H * Vd, E, 1.5), mix + "b": mat(H, E, 1.5), mix + "a": mat(H, E, 1.5), mix + "dt_bias": rnd(H, scale=1.5, mean=-3.0), mix + "A_log": rnd(H, scale=1.0),
                      mix + "norm": rnd(Vd, scale=0.2, mean=1.0)})
        elif s["type"] == "attention":
            G = m["kv_heads"]
            sharp = (2.5 / (m["scale"] * D ** 0.5)) ** 0.5          # scores of a few units, so that single keys count
            for n, rows, gain in (("q", H * D, sharp), ("k", G * D, sharp), ("v", G * Vd, 1.5)):
                w.update({mix + n: mat(rows, E, gain), mix + n + ".b": rnd(rows, scale=0.4)})
            if m["v_mix"]:
                w[mix + "vmix"] = rnd(1, scale=0.2, mean=0.5)[0]
        else:
            R, P, Q = m["kv_rank"], m["rot_dim"], m["q_rank"]
            sharp = 2.5 / (m["scale"] * (D + P) ** 0.5)
            w.update({mix + "dq": mat(Q, E), mix + "dq.norm": rnd(Q, scale=0.3, mean=1.0), mix + "uq": mat(H * (D + P), Q, sharp), mix + "dkv": mat(R + P, E), mix + "dkv.norm": rnd(R, scale=0.3, mean=1.0),
                      mix + "uk": mat(H * D, R), mix + "uv": mat(H * Vd, R)})
        w[mix + "o"] = mat(E, H * Vd)
        if s["mlp"] is not None:
            ff = s["mlp"]["ff"]
            w.update({p + "mlp.up": mat(ff, E), p + "mlp.down": mat(E, ff, 0.7), p + "mlp.act": rnd(2)})
    return w


def weights(cfg: dict, seed: int = 0) -> dict[str, torch.Tensor]:
    g = torch.Generator().manual_seed(seed)

    def rnd(*shape, scale=1.0, mean=0.0):
        return (torch.randn(*shape, generator=g) * scale + mean).to(torch.bfloat16)

    def mat(n, k, gain=1.0):
        return rnd(n, k, scale=gain / k ** 0.5)
    if cfg["architecture"] == "Nifalorn":
        return nifalorn_weights(cfg, g, rnd, mat)
    if cfg["architecture"] == "Rigalorn":
        return rigalorn_weights(cfg, g, rnd, mat)
    E, V = cfg["width"], cfg["vocab"]
    w = {"embed": rnd(V, E), "head": mat(V, E, 2.0), "final.norm": rnd(E, scale=0.2, mean=1.0)}
    if cfg["architecture"] == "Vozinex":
        w["final.norm.b"] = rnd(E, scale=0.2)
        for i, s in enumerate(cfg["layers"]):
            p, m = f"l{i}.", s["mixer"]
            H, G, D, Vd = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
            sharp = (2.5 / (m["scale"] * D ** 0.5)) ** 0.5          # scores of a few units, so that single keys count
            w.update({p + "norm1": rnd(E, scale=0.2, mean=1.0), p + "norm1.b": rnd(E, scale=0.2), p + "mix.q": mat(H * D, E), p + "mix.k": mat(G * D, E), p + "mix.v": mat(G * Vd, E, 1.5),
                      p + "mix.q.norm": rnd(H * D, scale=0.2, mean=1.0) * sharp, p + "mix.k.norm": rnd(G * D, scale=0.2, mean=1.0) * sharp, p + "mix.o": mat(E, H * Vd)})
            w[p + "mix.o"][:CODE] = 0
            if s["mlp"]:
                n, ff = s["mlp"]["router"]["experts"], s["mlp"]["expert"]["ff"]
                w.update({p + "norm2": rnd(E, scale=0.2, mean=1.0), p + "norm2.b": rnd(E, scale=0.2)})
                w[p + "norm2"][:CODE], w[p + "norm2.b"][:CODE] = 1, 0
                for e in range(n):
                    w.update({p + f"mlp.e{e}.up": mat(ff, E), p + f"mlp.e{e}.down": mat(E, ff)})
                    w[p + f"mlp.e{e}.down"][:CODE] = 0
                signs = torch.tensor(list(itertools.combinations(range(CODE), CODE // 2)))
                r = torch.zeros(n, E)
                r[:, :CODE] = -0.5
                r.scatter_(1, signs[torch.randperm(len(signs), generator=g)[:n]], 0.5)
                w.update({p + "mlp.router": r.to(torch.bfloat16), p + "mlp.router.b": (torch.randperm(n, generator=g) * (0.6 / n)).to(torch.bfloat16)})
        w["embed"][:, :CODE] = (torch.randint(0, 2, (V, CODE), generator=g) * 8 - 4).to(torch.bfloat16)
        return w
    for i, s in enumerate(cfg["layers"]):
        p, m = f"l{i}.", s["mixer"]
        H, D, Vd = m["heads"], m["dim"], m["vdim"]
        w[p + "norm1"] = rnd(E, scale=0.2, mean=0.7)
        if s["type"] == "hgrn2":
            lower = torch.rand(H * D, generator=g) * 0.9
            lower[torch.rand(H * D, generator=g) < 0.3] = 0.0
            w.update({p + "mix.q": mat(H * D, E, 1.5), p + "mix.f": mat(H * D, E, 1.5), p + "mix.f.b": rnd(H * D, scale=2.5, mean=2.0),
                      p + "mix.lower": lower.to(torch.bfloat16), p + "mix.v": mat(H * Vd, E), p + "mix.norm": rnd(Vd, scale=0.2, mean=1.0),
                      p + "mix.o": mat(E, H * Vd)})
        else:
            R = m["kv_rank"]
            w.update({p + "mix.q": mat(H * D, E, 2.0 / (m["scale"] * D ** 0.5)), p + "mix.dkv": mat(R, E), p + "mix.dkv.norm": rnd(R, scale=0.3, mean=1.0), p + "mix.uk": mat(H * D, R, 1.5),
                      p + "mix.uv": mat(H * Vd, R), p + "mix.g": mat(H, E), p + "mix.o": mat(E, H * Vd)})
        if s["mlp"]:
            ff = s["mlp"]["ff"]
            w.update({p + "norm2": rnd(E, scale=0.2, mean=0.7), p + "mlp.gate": mat(ff, E), p + "mlp.up": mat(ff, E), p + "mlp.down": mat(E, ff)})
    return w


def write(path: str, cfg: dict, w: dict[str, torch.Tensor]) -> str:
    os.makedirs(path, exist_ok=True)
    with open(os.path.join(path, "config.json"), "w") as f:
        json.dump(cfg, f)
    write_safetensors(os.path.join(path, "model.safetensors"), w)
    return path


def tokens(cfg: dict, n: int, seed: int = 0) -> list[int]:
    return torch.randint(0, cfg["vocab"], (n,), generator=torch.Generator().manual_seed(seed)).tolist()


def row_errors(got: torch.Tensor, want: torch.Tensor) -> torch.Tensor:
    """For every row the root mean square of the difference, relative to that of all wanted logits."""
    d = got.double().cpu() - want
    d = d - d.mean(-1, keepdim=True)
    return d.pow(2).mean(-1).sqrt() / want.pow(2).mean().sqrt()


def error(got: torch.Tensor, want: torch.Tensor) -> float:
    """The largest of the row errors."""
    return float(row_errors(got, want).max())


# ---- plain host forms of the kernels: bookkeeping tests without a GPU ------------------------------------------------------
def install_host_ops(monkeypatch):
    """Replace the kernel launches of ops.layers by plain fp32 code, so that engine, cache, state slots and scheduler run on the host."""
    from distributed_llm_pipeline_b200.ops import layers as L

    def row_stage(x, K, Kp, eps, y=None, w1=None, groups1=1, h_out=None, w2=None, groups2=1, b2=None, e=None, pair=0, lam=0.0, g=None, gate=0, tail=None):
        return dict(x=x, K=K, Kp=Kp, eps=eps, y=y, w1=w1, groups1=groups1, h_out=h_out, w2=w2, groups2=groups2, b2=b2, e=e, pair=pair, lam=lam, g=g, gate=gate, tail=tail)

    def staged(st, T):
        if st["pair"]:
            a, b = st["x"][:T, :2 * st["K"]].float().view(T, -1, 2, st["pair"]).unbind(2)
            v = (a - st["lam"] * b).reshape(T, -1)
        else:
            v = st["x"][:T, :st["K"]].float()
        if st["gate"] == 2:
            v = v * plain.silu(st["g"][:T, :st["K"]])
        if st["y"] is not None:
            v = v + (st["y"][:T] if st["w1"] is None else plain.grouped_norm(st["y"][:T], st["w1"], st["groups1"], st["eps"]))
        if st["e"] is not None:
            v = v + st["e"][:T]
        if st["h_out"] is not None:
            st["h_out"][:T] = v
        if st["b2"] is not None:
            v = plain.layer_norm(v, st["w2"], st["b2"], st["eps"])
        elif st["w2"] is not None:
            v = plain.grouped_norm(v, st["w2"].repeat(st["K"] // st["w2"].numel()), st["groups2"], st["eps"])
        if st["gate"] in (1, 3):
            v = v * (plain.sigmoid if st["gate"] == 1 else plain.silu)(st["g"][:T, :st["K"]])
        v = torch.nn.functional.pad(v, (0, st["Kp"] - st["K"]))
        return v if st["tail"] is None else torch.cat([v, st["tail"][:T].to(v.dtype)], 1)

    def behind(r, act):
        if act in (L.OUT_GEGLU, L.OUT_SWIGLU):
            return (plain.gelu_tanh if act == L.OUT_GEGLU else plain.silu)(r[..., 0::2]) * r[..., 1::2]
        return torch.clamp(r, min=0) ** 2 if act == L.OUT_RELU2 else r

    def out_tail(bias=None, n2=1 << 30, out2=None, act=(0.0, 0.0)):
        return bias, n2, out2, act

    def product(x, w, out, act, tail=None):
        r = behind(x.float() @ w.float().T, act)
        if tail is not None:
            bias, n2, out2, (pos, neg) = tail
            r = r if bias is None else r + bias
            if n2 < r.shape[1]:
                z = r[:, n2:]
                out2[:r.shape[0], :z.shape[1]] = (z / 2 + torch.where(z > 0, pos * z * z, neg * (torch.expm1(z) - z))).to(out2.dtype)
                r = r[:, :n2]
        out[:r.shape[0], :r.shape[1]] = r.to(out.dtype)
        return out

    def stage_rows(st, xb, T):
        xb[:T, :st["Kp"]] = staged(st, T).to(xb.dtype)
        return xb

    def head_matmul(x, x_head, kx, w, N, out, out_head, T, gate=None):
        for h in range(w.shape[0]):
            r = x[:T, h * x_head:h * x_head + kx].float() @ w[h, :N, :kx].float().T
            if gate is not None:
                r = r * torch.sigmoid(gate[:T, h:h + 1])
            out[:T, h * out_head:h * out_head + N] = r.to(out.dtype)
        return out

    def embed(table, ids, h, T, scale=1.0):
        h[:T] = table[ids[:T].long(), :h.shape[1]].float() * scale

    def latent_write(proj, w, eps, R, slot, cache, T, rot=None, q=None, heads=0):
        rows = cache.view(-1, cache.shape[-1])
        rows[slot[:T].long(), :R] = (plain.rms(proj[:T, :R], eps) * w).to(cache.dtype)
        if rot is not None:
            pos, f, amp = rot
            P = 2 * len(f)
            rows[slot[:T].long(), R:R + P] = (amp * plain.rotate_pairs(proj[:T, None, R:R + P], f, pos[:T]))[:, 0].to(cache.dtype)
            for h in range(heads):
                part = q[:T, (h + 1) * q.shape[1] // heads - P:(h + 1) * q.shape[1] // heads]
                part.copy_(amp * plain.rotate_pairs(part[:, None], f, pos[:T])[:, 0])

    def scan(proj, fbias, lower, state, seg, seg_slot, n_seg, pos, out, chunks=None):
        _, H, D, V = state.shape
        for s in range(n_seg):
            (lo, hi), sl = seg.view(-1, 2)[s].tolist(), int(seg_slot[s])
            x = proj[lo:hi]
            q, f, v = x[:, :H * D], x[:, H * D:2 * H * D], x[:, 2 * H * D:]
            st = torch.zeros_like(state[sl]) if int(pos[lo]) == 0 else state[sl]
            o, st = plain.hgrn2_scan((q * torch.sigmoid(q)).reshape(-1, H, D), plain.hgrn2_gates(f + fbias, lower).reshape(-1, H, D), v.reshape(-1, H, V), st)
            out[lo:hi] = o.reshape(hi - lo, -1)
            state[sl] = st
        return out

    def ssd(rows, hpg, state, decay, log_decay, seg, seg_slot, n_seg, pos, out, act=False, steps=None, skip=None, chunks=None, conv=None, single=False):
        _, H, D, V = state.shape
        if conv is not None:
            x, w, b, ring = conv
            y = conv_rows(x, w, b, ring, seg, seg_slot, n_seg, 1, pos, torch.empty_like(x))
            n = D * H // hpg
            rows = y[:, -n:], y[:, -2 * n:-n], y[:, :H * V]
        for s in range(n_seg):
            (lo, hi), sl = seg.view(-1, 2)[s].tolist(), int(seg_slot[s])
            assert not single or hi - lo == 1
            q, k, v = (r[lo:hi, :n].float() for r, n in zip(rows, (D * H // hpg, D * H // hpg, H * V)))
            if act:
                q, k, v = plain.silu(q), plain.silu(k), plain.silu(v)
            q, k, v = q.reshape(hi - lo, -1, D).repeat_interleave(hpg, 1), k.reshape(hi - lo, -1, D).repeat_interleave(hpg, 1), v.reshape(hi - lo, H, V)
            f = decay.expand(hi - lo, H) if steps is None else None
            if steps is not None:
                dt, f = plain.mamba2_steps(steps[0][lo:hi, :H], steps[1], torch.log(-log_decay))
                k = k * dt[:, :, None]
            o, state[sl] = plain.decayed_scan(q, k, v, f, torch.zeros_like(state[sl]) if int(pos[lo]) == 0 else state[sl])
            out[lo:hi] = (o + (skip[:, None] * v if skip is not None else 0)).reshape(hi - lo, -1)
        return out

    def delta(rows, hpg, state, a, b, log_decay, dt_bias, seg, seg_slot, n_seg, pos, out, unit_eps, chunks=None, conv=None, single=False):
        _, H, D, V = state.shape
        n = D * H // hpg
        assert unit_eps == 1e-6
        if conv is not None:
            y = conv_rows(*conv, seg, seg_slot, n_seg, 1, pos, torch.empty_like(conv[0]))
            rows = y, y[:, n:], y[:, 2 * n:]
        for s in range(n_seg):
            (lo, hi), sl = seg.view(-1, 2)[s].tolist(), int(seg_slot[s])
            assert not single or hi - lo == 1
            q, k, v = (r[lo:hi, :m].float().reshape(hi - lo, -1, w) for r, m, w in zip(rows, (n, n, H * V), (D, D, V)))
            q, k = (plain.unit(x).repeat_interleave(hpg, 1) for x in (q, k))
            f = torch.exp(log_decay * plain.softplus(a[lo:hi, :H] + dt_bias))
            o, state[sl] = plain.delta_scan(q * D ** -0.5, k, v, f, plain.sigmoid(b[lo:hi, :H]), torch.zeros_like(state[sl]) if int(pos[lo]) == 0 else state[sl])
            out[lo:hi, :H * V] = o.reshape(hi - lo, -1)
        return out

    def conv_rows(x, w, b, ring, seg, seg_slot, n_seg, longest, pos, out):
        taps, ch = w.shape
        for s in range(n_seg):
            (lo, hi), sl = seg.view(-1, 2)[s].tolist(), int(seg_slot[s])
            assert hi - lo <= longest
            p0 = int(pos[lo])
            before = torch.stack([ring[sl, p % taps] if p >= 0 else torch.zeros(ch) for p in range(p0 - taps + 1, p0)]) if taps > 1 else torch.zeros(0, ch)
            out[lo:hi, :ch] = plain.silu(plain.causal_conv(x[lo:hi, :ch], w.T, torch.zeros(ch) if b is None else b, before))
            for t in range(max(lo, hi - taps), hi):
                ring[sl, (p0 + t - lo) % taps] = x[t, :ch]
        return out

    def attention(q, cache, block_table, tok_slot, pos, tile_row0, tile_rows, n_tiles, bm, H, T, scale, out, n_splits=1, workspace=None, window=1 << 30):
        page, Rc = cache.shape[-2], cache.shape[-1]
        rows = cache.view(-1, Rc)
        seen = torch.zeros(T * H, dtype=torch.bool)
        for i in range(n_tiles):
            r0, n = int(tile_row0[i]), int(tile_rows[i])
            assert len({int(tok_slot[r // H]) for r in range(r0, r0 + n)}) == 1 and n <= bm and not seen[r0:r0 + n].any()
            seen[r0:r0 + n] = True
        assert seen.all()
        for t in range(T):
            k = torch.arange(max(0, int(pos[t]) + 1 - window), int(pos[t]) + 1)
            c = rows[block_table[int(tok_slot[t]), k // page].long() * page + k % page].float()
            p = torch.softmax(q[t].view(H, Rc).float() @ c.T * scale, -1)
            out[t] = (p @ c)[:, :out.shape[1] // H].reshape(-1).to(out.dtype)
        return out

    def choose(logits, r):
        z = logits[:, :r.n]
        if r.sigmoid:
            return plain.group_route(z, torch.eye(r.n), r.bias, r.top, r.groups, r.keep, r.scale)
        return plain.route(z, torch.eye(r.n), r.bias, r.top)

    def route(logits, rule, ids, weights, T):
        i, p = choose(logits[:T], rule)
        ids[:], weights[:] = i.reshape(-1).to(torch.int32), p.reshape(-1)

    def expert_matvec(st, logits, rule, w, rows, out, T, down, act=L.OUT_RELU2, shared=None):
        assert T <= 4
        top = rule.top
        i, p = choose(logits[:T], rule)
        x, m = staged(st, T * top if down else T), w.view(rule.n, rows, -1).float()
        if shared is not None and not down:
            r = behind(x @ shared[0].float().T, act)
            shared[1][:T, :r.shape[1]] = r
        for t in range(T):
            for j in range(top):
                y = m[i[t, j]] @ x[t * top + j if down else t]
                if not down:
                    y = behind(y, act)
                    out[t * top + j, :y.numel()] = y
                elif j == 0:
                    out[t, :rows] = p[t, j] * y
                else:
                    out[t, :rows] += p[t, j] * y
            if shared is not None and down:
                out[t, :rows] += plain.sigmoid(logits[t, rule.n]) * (shared[0].float() @ shared[1][t].float())

    def expert_plan(ids, n_expert, tile, plan):
        order = torch.sort(ids, stable=True).indices
        plan.src[:ids.numel()] = order.to(torch.int32)
        plan.pos[order] = torch.arange(ids.numel(), dtype=torch.int32)
        plan.sorted_ids = ids[order].long()

    def expert_gather(x, plan, top, n, out):
        out[:] = x[plan.src[:n].long() // top]
        return out

    def linear_grouped(xs, w, rows, n_expert, tile, plan, out, act=L.OUT_F32):
        out[:] = behind(torch.einsum("ak,ark->ar", xs.float(), w.view(n_expert, rows, -1)[plan.sorted_ids].float()), act).to(out.dtype)
        return out

    def expert_combine(y, plan, weights, T, top, out, shared=None):
        out[:T] = (y[plan.pos[:T * top].long()] * weights[:, None]).view(T, top, -1).sum(1)
        if shared is not None:
            out[:T] += plain.sigmoid(shared[1][:T, :1]) * shared[0][:T]

    def gqa_prepare(m, proj, kc, vc, block_table, tok_slot, pos, slot, q, T, mix=None):
        HD, GD, ps = m.H * m.D, m.G * m.maps * m.D, kc.shape[-2]
        q.zero_()

        def turn(x, p):
            if m.adjacent:
                return plain.rotate_pairs(x, m.inv_freq, p)
            a = p.float()[:, None, None] * m.inv_freq
            n, c, s = m.rot // 2, m.rot_scale * torch.cos(a), m.rot_scale * torch.sin(a)
            return torch.cat([x[..., :n] * c - x[..., n:2 * n] * s, x[..., n:2 * n] * c + x[..., :n] * s, x[..., 2 * n:]], -1)
        values = proj[:T, HD + GD:HD + GD + m.G * m.V]
        if mix is not None:
            first, lam = mix
            if lam is None:
                first.copy_(values)
            else:
                values = (1 - lam) * values + lam * first
        for t in range(T):
            a, b = (turn((plain.rms(x, m.eps) * n if n is not None else x).view(1, -1, m.D), pos[t:t + 1])
                    for x, n in ((proj[t, :HD], m.q_norm), (proj[t, HD:HD + GD], m.k_norm)))
            q[t].view(m.H, m.Dc)[:, :m.D] = a[0]
            page, off = int(slot[t]) // ps, int(slot[t]) % ps
            kc[page, :, off, :m.D] = b[0]
            vc[page, :, off, :m.V] = values[t].view(m.G, m.V)

    def gqa_attention(m, q, kc, vc, block_table, tok_slot, pos, tiles, bm, n_splits, out, T):
        row0, rows, n = tiles
        ps, seen = kc.shape[-2], []
        for i in range(n):
            lo, c = int(row0[i]), int(rows[i])
            assert 1 <= c <= bm // min(m.R, bm) and len(set(tok_slot[lo:lo + c].tolist())) == 1 and int(pos[lo + c - 1]) - int(pos[lo]) == c - 1
            for t in range(lo, lo + c):
                seen.append(t)
                p = int(pos[t])
                j = torch.arange(p + 1)
                pages = block_table[int(tok_slot[t]), j // ps].long()
                k, v = kc[pages, :, j % ps, :m.D].float(), vc[pages, :, j % ps, :m.V].float()
                qp = torch.nn.functional.pad(q[t].view(1, m.H, m.Dc)[..., :m.D].float(), (0, 0, 0, 0, p, 0))
                seen_keys = plain.window_mask(p + 1, m.window, m.keep) & (plain.chunk_mask(p + 1, m.chunk) if m.chunk else True)
                o = torch.stack([plain.masked_softmax_attention(qp[:, i::m.maps], k[:, i::m.maps], v, m.scale, seen_keys)[p] for i in range(m.maps)], 1)
                out[t, :m.H * m.V] = o.reshape(-1).to(out.dtype)
        assert len(seen) == len(set(seen))
        return out
    for name, fn in dict(route=route, expert_matvec=expert_matvec, expert_plan=expert_plan, expert_gather=expert_gather, linear_grouped=linear_grouped,
                         expert_combine=expert_combine, ssd=ssd, delta=delta, out_tail=out_tail, conv_rows=conv_rows, conv_args=lambda *a: a, gqa_prepare=gqa_prepare, gqa_attention=gqa_attention).items():
        monkeypatch.setattr(L, name, fn)
    for name, fn in dict(row_stage=row_stage, stage_rows=stage_rows, head_matmul=head_matmul, embed=embed, latent_write=latent_write, hgrn2=scan,
                         latent_attention=attention, matvec=lambda st, w, out, T, act=0, tail=None: product(staged(st, T), w, out, act, tail),
                         linear=lambda x, w, out, act=0, tail=None: product(x, w, out, act, tail)).items():
        monkeypatch.setattr(L, name, fn)
