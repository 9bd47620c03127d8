"""Helpers of the Gapidra tests: small configurations that differ from each other in every size, in the layer order, in their
windows and constants and in which optional parts they have, and a driver that feeds sequences to an op in given portions.
Checkpoints, engines and schedule replay are the ones of kofadra_util."""
import torch

from kofadra_util import make_engine, rel_err, replay, save_checkpoint, tokens  # noqa: F401

import gapidra_ref as R

# rel_err bounds: the worst position in fp32 (the engine stands at 1e-6 .. 3e-6 on these geometries), the 80th percentile in
# bf16 (4e-3 .. 1e-2)
TOL = {"float32": 2e-5, "bfloat16": 3e-2}


def dense(ff):
    return {"kind": "dense", "ff": ff}


def yarn(factor, original, fast, slow):
    return {"factor": factor, "original": original, "fast": fast, "slow": slow}


def _mixer(m, size, dims, base, scaling):
    if size:
        m["mask"] = {"size": size}
    if dims is not None:
        m["rot"] = {"dims": dims, "base": base}
        if scaling:
            m["rot"]["scaling"] = scaling
    return m


def latent(heads, dim, rot_dim, vdim, kv_rank, scale, size=0, base=10000.0, mlp=None):
    return {"type": "latent_attention", "mlp": mlp,
            "mixer": _mixer({"heads": heads, "dim": dim, "rot_dim": rot_dim, "vdim": vdim, "kv_rank": kv_rank, "scale": scale},
                            size, rot_dim, base, None)}


def sigmoid(heads, kv_heads, dim, vdim, scale, size=0, dims=None, base=10000.0, scaling=None, mlp=None):
    return {"type": "attention", "mlp": mlp,
            "mixer": _mixer({"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "scale": scale}, size, dims, base, scaling)}


def config(width, vocab, layers, eps=1e-5, embed_scale=1.0):
    return {"architecture": "Gapidra", "vocab": vocab, "width": width, "layers": layers, "norm": {"eps": eps},
            "embedding": {"scale": embed_scale}}


def cfg_a():      # odd vocabulary, G < H, windows below and above a page, a layer without feed-forward, vdim on both sides of dim
    return config(64, 97, [sigmoid(4, 1, 24, 16, 0.3, size=9, dims=12, base=500.0, scaling=yarn(4.0, 300, 8.0, 1.0), mlp=dense(40)),
                           latent(3, 16, 8, 20, 24, 0.2, size=17, base=300.0, mlp=dense(56)),
                           latent(2, 8, 4, 36, 12, 0.3, size=5, base=77.0),
                           sigmoid(3, 3, 16, 28, 0.25, size=33, dims=16, base=900.0, mlp=dense(24))], embed_scale=2.5)


def cfg_b():      # no window at all, one head, nothing turns in one layer, no rotation entry in another
    return config(48, 130, [latent(1, 12, 6, 8, 20, 0.4, base=50.0),
                            sigmoid(2, 2, 16, 16, 0.2, dims=0, mlp=dense(32)),
                            sigmoid(6, 2, 8, 24, 0.5, mlp=dense(20)),
                            latent(5, 8, 12, 12, 32, 0.25, base=2e4, mlp=dense(48))], eps=1e-6)


def cfg_c():      # windows of one token, of a page, of a page + 1; head sizes that are no power of two; two scalings
    return config(80, 64, [sigmoid(5, 5, 40, 12, 0.2, size=1, dims=20, base=1e3, scaling=yarn(16.0, 64, 4.0, 0.5), mlp=dense(48)),
                           latent(2, 40, 20, 12, 28, 0.15, size=16, base=1e6, mlp=dense(16)),
                           sigmoid(4, 2, 24, 40, 0.2, size=17, dims=8, base=2e3, scaling=yarn(2.5, 128, 6.0, 1.5)),
                           latent(4, 4, 8, 24, 16, 0.3, size=1, base=1e2, mlp=dense(64)),
                           sigmoid(1, 1, 20, 20, 0.3, size=16, dims=20, base=3e4, mlp=dense(12))], embed_scale=0.7)


def cfg_d():      # no size a multiple of four
    return config(30, 51, [latent(3, 6, 6, 10, 14, 0.4, size=5, base=30.0, mlp=dense(22)),
                           sigmoid(6, 3, 6, 10, 0.5, size=7, dims=2, base=9.0, mlp=dense(14)),
                           sigmoid(1, 1, 14, 2, 0.3, size=18, dims=6, base=99.0, scaling=yarn(3.0, 50, 2.0, 0.5))], embed_scale=1.3)


def cfg_e():      # sizes the tensor-core kernels take in bf16: heads of 32 and 64, latents of 64 + 16 and 256 + 48
    return config(96, 200, [latent(6, 32, 16, 32, 64, 0.14, size=50, base=4e4, mlp=dense(96)),
                            sigmoid(4, 2, 64, 32, 0.125, size=41, dims=32, base=2e5, scaling=yarn(8.0, 512, 16.0, 1.0), mlp=dense(64)),
                            latent(3, 48, 48, 16, 256, 0.1, size=90, base=1e4, mlp=dense(32)),
                            sigmoid(2, 1, 32, 96, 0.2, size=64, dims=16, base=1e5)], embed_scale=3.0)


def cfg_f():      # eight query heads on one key head of 128, a latent of 128 + 32 under twenty heads, no window in the latent layer
    return config(128, 90, [sigmoid(8, 1, 128, 64, 0.09, size=50, dims=96, base=1e5, mlp=dense(96)),
                            latent(20, 16, 32, 16, 128, 0.14, base=1e4, mlp=dense(72)),
                            latent(4, 24, 8, 80, 128, 0.18, size=130, base=5e3)], embed_scale=4.0)


CONFIGS = {"a": cfg_a, "b": cfg_b, "c": cfg_c, "d": cfg_d, "e": cfg_e, "f": cfg_f}


def oracle_logits(cfg: dict, weights, toks):
    return R.forward(cfg, weights, toks)


# ------------------------------------------------------------------------------------------------ ops in portions
def pages(n_pages: int, seed: int):
    """A shuffled order of the pool's pages."""
    return torch.randperm(n_pages, generator=torch.Generator().manual_seed(seed)).tolist()


def feed(cuda, seqs, tables, bs, schedule, fn):
    """seqs: one [T_s, P] tensor of input rows per sequence; tables: the pages of each; schedule: steps of [(sequence, rows)].
    fn(rows [n, P], batch, positions, slots) -> [n, ...] runs one step on the device.  Returns one output per sequence."""
    from b200attn import ops
    i32 = lambda v: torch.tensor(v, dtype=torch.int32, device=cuda)      # noqa: E731
    at, outs = [0] * len(seqs), [[] for _ in seqs]
    width = max(len(t) for t in tables)
    for step in schedule:
        rows, cu, ctx, tab, pos, slots = [], [0], [], [], [], []
        for s, n in step:
            lo, hi = at[s], at[s] + n
            assert hi <= seqs[s].shape[0]
            rows.append(seqs[s][lo:hi])
            cu.append(cu[-1] + n), ctx.append(lo), tab.append(tables[s] + [0] * (width - len(tables[s])))
            pos += range(lo, hi)
            slots += [tables[s][p // bs] * bs + p % bs for p in range(lo, hi)]
            at[s] = hi
        batch = ops.SeqBatch(i32(cu), i32(ctx), i32(tab), None, len(step), cu[-1])
        o = fn(torch.cat(rows).to(cuda), batch, i32(pos), torch.tensor(slots, dtype=torch.int64, device=cuda))
        for k, (s, n) in enumerate(step):
            outs[s].append(o[cu[k]:cu[k + 1]].clone())
    assert all(a == q.shape[0] for a, q in zip(at, seqs)), "the schedule must use up every sequence"
    return [torch.cat(o) for o in outs]
