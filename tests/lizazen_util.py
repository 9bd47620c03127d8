"""Helpers of the Lizazen tests: small configurations that differ from each other in every size, in the layer order, in their
windows and constants and in which optional parts they have, and a driver that feeds sequences to an op in given portions.
Checkpoints, engines and schedule replay are the ones of kofadra_util."""
import torch

from gapidra_util import pages  # noqa: F401
from kofadra_util import make_engine, rel_err, replay, save_checkpoint, tokens  # noqa: F401

import lizazen_ref as R

# rel_err bounds: the worst position in fp32 (the engine stands at 5e-7 .. 6e-6 on these geometries), the 80th percentile in
# bf16 (6e-3 .. 2e-2)
TOL = {"float32": 2e-5, "bfloat16": 4e-2}


def dense(ff, limit):
    return {"kind": "dense", "ff": ff, "limit": limit}


def moe(experts, top, ff, shared=0):
    f = {"kind": "moe", "expert": {"ff": ff}, "router": {"experts": experts, "top": top}}
    if shared:
        f["shared"] = {"ff": shared}
    return f


def zones(factor, low, high, original):
    return {"factor": factor, "low": low, "high": high, "original": original}


def rot(dims, base, scaling=None):
    r = {"dims": dims, "base": base}
    if scaling:
        r["scaling"] = scaling
    return r


def _with(m, mask, rotation):
    m["mask"] = mask
    if rotation:
        m["rot"] = rotation
    return m


def window(heads, kv_heads, dim, scale, size, rotation=None, cap=None, mlp=None):
    m = {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": dim, "scale": scale}
    if cap:
        m["softcap"] = cap
    return {"type": "attention", "mlp": mlp, "mixer": _with(m, {"size": size}, rotation)}


def diff(heads, kv_heads, dim, vdim, scale, part, size, keep=0, rotation=None, mlp=None):
    m = {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "scale": scale, "diff": part}
    return {"type": "attention_2", "mlp": mlp, "mixer": _with(m, {"size": size, "keep_first": keep}, rotation)}


def pair(left, right, mlp=None):
    return {"type": "parallel", "mlp": mlp, "mixer": {"left": left, "right": right}}


def chunk(heads, kv_heads, dim, vdim, scale, size, rotation=None):
    return _with({"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "scale": scale}, {"size": size}, rotation)


def retention(dim, vdim, decay, rotation=None):
    m = {"heads": len(decay), "dim": dim, "vdim": vdim, "decay": decay}
    if rotation:
        m["rot"] = rotation
    return m


def config(width, vocab, layers, bigram=(31, 17, 5), eps=1e-5):
    c = {"architecture": "Lizazen", "vocab": vocab, "width": width, "layers": layers, "norm": {"eps": eps}, "embedding": {}}
    if bigram:
        c["embedding"]["bigram"] = dict(zip(("buckets", "mul_prev", "mul_cur"), bigram))
    return c


def cfg_a():      # odd vocabulary, G < H, windows below and above a page, vdim on both sides of dim, a layer without feed-forward
    return config(64, 97, [pair(chunk(4, 2, 24, 16, 0.25, 24, rot(12, 300.0)), retention(16, 24, [0.5, 0.95, 1.0], rot(8, 90.0)), moe(5, 2, 24, 40)),
                           window(4, 1, 24, 0.3, 9, rot(12, 500.0, zones(4.0, 1.0, 4.0, 300)), 5.0, dense(40, 0.7)),
                           diff(3, 1, 16, 40, 0.3, 0.2, 17, 5, rot(16, 77.0)),
                           diff(2, 2, 8, 4, 0.5, 0.6, 5, 40, rot(4, 30.0), moe(3, 1, 16))])


def cfg_b():      # no rotation anywhere, no cap, no kept tokens, every expert chosen, no shared expert, no bigram table
    return config(48, 130, [diff(1, 1, 12, 20, 0.4, 0.35, 64, mlp=dense(36, 3.0)),
                            window(2, 2, 16, 0.2, 200, mlp=moe(2, 2, 20)),
                            pair(chunk(6, 2, 8, 24, 0.5, 40), retention(20, 12, [0.9, 0.8]), dense(20, 0.1))], bigram=None, eps=1e-6)


def cfg_c():      # windows and chunks of one token, of a page, of a page + 1; head sizes that are no power of two; other scalings
    return config(80, 64, [window(5, 5, 40, 0.2, 1, rot(20, 1e3, zones(16.0, 0.5, 2.0, 64)), 2.0, moe(4, 3, 24, 8)),
                           diff(2, 2, 20, 12, 0.15, 0.8, 16, 1, rot(6, 1e4), dense(48, 1.5)),
                           pair(chunk(4, 2, 24, 40, 0.2, 17, rot(8, 2e3)), retention(40, 8, [0.99, 0.7, 0.97, 0.999], rot(40, 1e3)), moe(6, 1, 12, 64)),
                           pair(chunk(1, 1, 20, 20, 0.3, 1), retention(28, 12, [0.95]), dense(12, 7.0)),
                           window(4, 2, 24, 0.3, 17, rot(24, 3e4), 30.0, dense(16, 2.0)),
                           pair(chunk(2, 1, 12, 28, 0.3, 16, rot(12, 50.0)), retention(12, 28, [0.6, 0.9], rot(2, 7.0)))],
                  bigram=(1, 3, 0), eps=1e-4)


def cfg_d():      # no size a multiple of four
    return config(30, 51, [diff(3, 3, 6, 10, 0.4, 0.45, 7, 3, rot(6, 30.0), moe(7, 3, 22, 18)),
                           window(6, 3, 6, 0.5, 5, rot(2, 9.0, zones(3.0, 1.0, 8.0, 50)), 1.5, dense(14, 0.9)),
                           pair(chunk(1, 1, 14, 2, 0.3, 18, rot(6, 99.0)), retention(10, 6, [0.93, 0.5, 0.99], rot(10, 20.0)), dense(26, 5.0))],
                  bigram=(10, 7, 13))


def cfg_e():      # sizes the tensor-core prompt kernel takes in bf16, values of 192 beside keys of 64
    return config(96, 200, [window(4, 2, 64, 0.125, 50, rot(32, 2e5, zones(8.0, 1.0, 4.0, 512)), 20.0, moe(8, 2, 32, 48)),
                            diff(4, 2, 32, 64, 0.18, 0.3, 41, 20, rot(8, 4e4), dense(96, 1.0)),
                            pair(chunk(2, 1, 64, 192, 0.12, 90, rot(16, 1e5)), retention(32, 64, [0.98, 0.995], rot(32, 1e4)), moe(4, 1, 64, 32))],
                  bigram=(499, 1009, 31))


def cfg_f():      # eight query heads on one key head of 128; twelve maps on one value head of 128; keys of 96 under values of 256
    return config(128, 90, [window(8, 1, 128, 0.09, 60, rot(96, 1e5), 50.0, dense(96, 4.0)),
                            pair(chunk(2, 2, 96, 256, 0.1, 48, rot(96, 1e4)), retention(96, 32, [0.97, 0.999, 1.0], rot(64, 1e3)), moe(3, 3, 40, 24)),
                            diff(6, 1, 64, 128, 0.12, 0.25, 130, 16, rot(64, 5e3), moe(16, 4, 16, 16))], bigram=(64, 5, 1))


CONFIGS = {"a": cfg_a, "b": cfg_b, "c": cfg_c, "d": cfg_d, "e": cfg_e, "f": cfg_f}


def oracle_logits(cfg: dict, weights, toks):
    return R.forward(cfg, weights, toks)


# ------------------------------------------------------------------------------------------------ ops in portions
def feed(cuda, seqs, schedule, fn, bs=16, tables=None, slots=None):
    """seqs: one tensor of input rows per sequence; schedule: steps of [(sequence, rows)]; tables: the pages of each sequence,
    slots: its state slot.  fn(rows [n, ...], batch, positions, cache slots) -> [n, ...] runs one step on the device.  Returns one
    output per sequence."""
    from b200attn import ops
    i32 = lambda v: torch.tensor(v, dtype=torch.int32, device=cuda)      # noqa: E731
    at, outs = [0] * len(seqs), [[] for _ in seqs]
    width = max(len(t) for t in tables) if tables else 1
    for step in schedule:
        rows, cu, ctx, tab, pos, where = [], [0], [], [], [], []
        for s, n in step:
            lo, hi = at[s], at[s] + n
            assert hi <= seqs[s].shape[0]
            rows.append(seqs[s][lo:hi])
            cu.append(cu[-1] + n), ctx.append(lo)
            pos += range(lo, hi)
            if tables:
                tab.append(tables[s] + [0] * (width - len(tables[s])))
                where += [tables[s][p // bs] * bs + p % bs for p in range(lo, hi)]
            at[s] = hi
        batch = ops.SeqBatch(i32(cu), i32(ctx), i32(tab) if tables else None, i32([slots[s] for s, _ in step]) if slots else None,
                             len(step), cu[-1])
        o = fn(torch.cat(rows).to(cuda), batch, i32(pos), torch.tensor(where, dtype=torch.int64, device=cuda))
        for k, (s, n) in enumerate(step):
            outs[s].append(o[cu[k]:cu[k + 1]].clone())
    assert all(a == q.shape[0] for a, q in zip(at, seqs)), "the schedule must use up every sequence"
    return [torch.cat(o) for o in outs]
