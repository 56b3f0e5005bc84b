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
    "attention": config(80, 64, 5, [latent(4, 16, 24, 32, 0.4, 40), latent(49, 8, 4, 64, 0.4)]),
}


CODE = 8     # Vozinex: leading dimensions that only the embedding writes and only the routers read, as signs, so that no routing is a close call
             # (a model in bf16 would choose other experts there, and the comparison with exact arithmetic would say nothing)


def weights(cfg: dict, seed: int = 0) -> dict[str, torch.Tensor]:
    g = torch.Generator().manual_seed(seed)

    def rnd(*shape, scale=1.0, mean=0.0):
        return (torch.randn(*shape, generator=g) * scale + mean).to(torch.bfloat16)

    def mat(n, k, gain=1.0):
        return rnd(n, k, scale=gain / k ** 0.5)
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


def error(got: torch.Tensor, want: torch.Tensor) -> float:
    """Largest over the rows: root mean square of the difference, relative to that of all wanted logits."""
    d = got.double().cpu() - want
    d = d - d.mean(-1, keepdim=True)
    return float(d.pow(2).mean(-1).sqrt().max() / want.pow(2).mean().sqrt())


# ---- plain host forms of the kernels: bookkeeping tests without a GPU ------------------------------------------------------
def install_host_ops(monkeypatch):
    """Replace the kernel launches of ops.layers by plain fp32 code, so that engine, cache, state slots and scheduler run on the host."""
    from distributed_llm_pipeline_b200.ops import layers as L

    def row_stage(x, K, Kp, eps, y=None, w1=None, groups1=1, h_out=None, w2=None, groups2=1, b2=None, e=None):
        return dict(x=x, K=K, Kp=Kp, eps=eps, y=y, w1=w1, groups1=groups1, h_out=h_out, w2=w2, groups2=groups2, b2=b2, e=e)

    def staged(st, T):
        v = st["x"][:T, :st["K"]].float()
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

    def route(logits, bias, n_expert, top, ids, weights, T):
        i, p = plain.route(logits[:T], torch.eye(n_expert), bias, top)
        ids[:], weights[:] = i.reshape(-1).to(torch.int32), p.reshape(-1)

    def expert_matvec(st, logits, bias, n_expert, top, w, rows, out, T, down):
        assert T <= 4
        i, p = plain.route(logits[:T], torch.eye(n_expert), bias, top)
        x, m = staged(st, T * top if down else T), w.view(n_expert, rows, -1).float()
        for t in range(T):
            for j in range(top):
                y = m[i[t, j]] @ x[t * top + j if down else t]
                if not down:
                    out[t * top + j, :rows] = torch.clamp(y, min=0) ** 2
                elif j == 0:
                    out[t, :rows] = p[t, j] * y
                else:
                    out[t, :rows] += p[t, j] * y

    def expert_plan(ids, n_expert, tile, plan):
        order = torch.sort(ids, stable=True).indices
        plan.src[:ids.numel()] = order.to(torch.int32)
        plan.pos[order] = torch.arange(ids.numel(), dtype=torch.int32)
        plan.sorted_ids = ids[order].long()

    def expert_gather(x, plan, top, n, out):
        out[:] = x[plan.src[:n].long() // top]
        return out

    def linear_grouped(xs, w, rows, n_expert, tile, plan, out, relu2=False):
        y = torch.einsum("ak,ark->ar", xs.float(), w.view(n_expert, rows, -1)[plan.sorted_ids].float())
        out[:] = (torch.clamp(y, min=0) ** 2 if relu2 else y).to(out.dtype)
        return out

    def expert_combine(y, plan, weights, T, top, out):
        out[:T] = (y[plan.pos[:T * top].long()] * weights[:, None]).view(T, top, -1).sum(1)

    def gqa_prepare(m, proj, kc, vc, block_table, tok_slot, pos, slot, q, T):
        HD, GD, ps = m.H * m.D, m.G * m.D, kc.shape[-2]
        q.zero_()
        for t in range(T):
            a, b = (plain.rotate_half((plain.rms(x, m.eps) * n).view(1, -1, m.D), m.rot, m.base, pos[t:t + 1])
                    for x, n in ((proj[t, :HD], m.q_norm), (proj[t, HD:HD + GD], m.k_norm)))
            q[t].view(m.H, m.Dc)[:, :m.D] = a[0]
            page, off = int(slot[t]) // ps, int(slot[t]) % ps
            kc[page, :, off, :m.D] = b[0]
            vc[page, :, off, :m.V] = proj[t, HD + GD:].view(m.G, m.V)

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
                o = plain.masked_softmax_attention(torch.nn.functional.pad(q[t].view(1, m.H, m.Dc)[..., :m.D].float(), (0, 0, 0, 0, p, 0)), k, v, m.scale,
                                                   plain.window_mask(p + 1, m.window, m.keep))[p]
                out[t, :m.H * m.V] = o.reshape(-1).to(out.dtype)
        assert len(seen) == len(set(seen))
        return out
    for name, fn in dict(route=route, expert_matvec=expert_matvec, expert_plan=expert_plan, expert_gather=expert_gather, linear_grouped=linear_grouped,
                         expert_combine=expert_combine, gqa_prepare=gqa_prepare, gqa_attention=gqa_attention).items():
        monkeypatch.setattr(L, name, fn)
    for name, fn in dict(row_stage=row_stage, stage_rows=stage_rows, head_matmul=head_matmul, embed=embed, latent_write=latent_write, hgrn2=scan,
                         latent_attention=attention, matvec=lambda st, w, out, T, geglu=False: product(staged(st, T), w, out, geglu),
                         linear=lambda x, w, out, geglu=False: product(x, w, out, geglu)).items():
        monkeypatch.setattr(L, name, fn)
