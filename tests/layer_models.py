"""Small random layer-list models for the tests, and a way to run the engine's bookkeeping without a GPU."""
from __future__ import annotations

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
    "attention": config(80, 64, 5, [latent(4, 16, 24, 32, 0.4, 40), latent(49, 8, 4, 64, 0.4)]),
}


def weights(cfg: dict, seed: int = 0) -> dict[str, torch.Tensor]:
    g = torch.Generator().manual_seed(seed)

    def rnd(*shape, scale=1.0, mean=0.0):
        return (torch.randn(*shape, generator=g) * scale + mean).to(torch.bfloat16)

    def mat(n, k, gain=1.0):
        return rnd(n, k, scale=gain / k ** 0.5)
    E, V = cfg["width"], cfg["vocab"]
    w = {"embed": rnd(V, E), "head": mat(V, E, 2.0), "final.norm": rnd(E, scale=0.2, mean=1.0)}
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


def error(got: torch.Tensor, want: torch.Tensor) -> float:
    """Largest over the rows: root mean square of the difference, relative to that of all wanted logits."""
    d = got.double().cpu() - want
    d = d - d.mean(-1, keepdim=True)
    return float(d.pow(2).mean(-1).sqrt().max() / want.pow(2).mean().sqrt())


# ---- plain host forms of the kernels: bookkeeping tests without a GPU ------------------------------------------------------
def install_host_ops(monkeypatch):
    """Replace the kernel launches of ops.layers by plain fp32 code, so that engine, cache, state slots and scheduler run on the host."""
    from distributed_llm_pipeline_b200.ops import layers as L

    def row_stage(x, K, Kp, eps, y=None, w1=None, groups1=1, h_out=None, w2=None, groups2=1):
        return dict(x=x, K=K, Kp=Kp, eps=eps, y=y, w1=w1, groups1=groups1, h_out=h_out, w2=w2, groups2=groups2)

    def staged(st, T):
        v = st["x"][:T, :st["K"]].float()
        if st["y"] is not None:
            v = v + plain.grouped_norm(st["y"][:T], st["w1"], st["groups1"], st["eps"])
            if st["h_out"] is not None:
                st["h_out"][:T] = v
        if st["w2"] is not None:
            v = plain.grouped_norm(v, st["w2"].repeat(st["K"] // st["w2"].numel()), st["groups2"], st["eps"])
        return torch.nn.functional.pad(v, (0, st["Kp"] - st["K"]))

    def product(x, w, out, geglu):
        r = x.float() @ w.float().T
        if geglu:
            r = plain.gelu_tanh(r[:, 0::2]) * r[:, 1::2]
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

    def embed(table, ids, h, T):
        h[:T] = table[ids[:T].long(), :h.shape[1]].float()

    def latent_write(proj, w, eps, R, slot, cache, T):
        rows = cache.view(-1, cache.shape[-1])
        rows[slot[:T].long(), :R] = (plain.rms(proj[:T, :R], eps) * w).to(cache.dtype)

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

    def attention(q, cache, block_table, tok_slot, pos, tile_row0, tile_rows, n_tiles, bm, H, T, scale, out, n_splits=1, workspace=None):
        page, Rc = cache.shape[-2], cache.shape[-1]
        rows = cache.view(-1, Rc)
        seen = torch.zeros(T * H, dtype=torch.bool)
        for i in range(n_tiles):
            r0, n = int(tile_row0[i]), int(tile_rows[i])
            assert len({int(tok_slot[r // H]) for r in range(r0, r0 + n)}) == 1 and n <= bm and not seen[r0:r0 + n].any()
            seen[r0:r0 + n] = True
        assert seen.all()
        for t in range(T):
            k = torch.arange(int(pos[t]) + 1)
            c = rows[block_table[int(tok_slot[t]), k // page].long() * page + k % page].float()
            p = torch.softmax(q[t].view(H, Rc).float() @ c.T * scale, -1)
            out[t] = (p @ c).reshape(-1).to(out.dtype)
        return out
    for name, fn in dict(row_stage=row_stage, stage_rows=stage_rows, head_matmul=head_matmul, embed=embed, latent_write=latent_write, hgrn2=scan,
                         latent_attention=attention, matvec=lambda st, w, out, T, geglu=False: product(staged(st, T), w, out, geglu),
                         linear=lambda x, w, out, geglu=False: product(x, w, out, geglu)).items():
        monkeypatch.setattr(L, name, fn)
