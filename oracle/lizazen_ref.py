"""Plain CPU restatement of the Lizazen decoder, one function per mechanism (test infrastructure only).

Everything runs in float64 on whole sequences; nothing here is shared with the product path under
vllm-backend-public_b200/ (which never imports this file).  `weights` maps the checkpoint's tensor names to tensors;
`cfg` is the parsed config.json dictionary.

Notation: T tokens, D model width, H query heads, G key/value heads, dk / dv per-head key and value sizes.
"""
from __future__ import annotations

import math
from typing import Callable, Dict, List, Optional

import torch

F64 = torch.float64


# ------------------------------------------------------------------------------------------------ norm, activations
def unit_rms(x, eps):
    """x / sqrt(mean(x^2) + eps) over the last axis."""
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps)


def rms_norm(x, w, eps):
    return unit_rms(x, eps) * w


def sigmoid(z):
    return 1.0 / (1.0 + torch.exp(-z))


def silu(z):
    return z * sigmoid(z)


def bounded_glu(g, u, limit: float):
    """Both inputs bounded: g' = min(g, limit), u' within +-limit; g' sigmoid(1.702 g') (u' + 1)."""
    g = torch.clamp(g, max=limit)
    u = torch.clamp(u, min=-limit, max=limit)
    return g * sigmoid(1.702 * g) * (u + 1.0)


# ------------------------------------------------------------------------------------------------ embedding
def bigram_row(prev: Optional[int], cur: int, b: dict) -> int:
    """Row of the bigram table for token `cur` behind token `prev` (None: the sequence's first token)."""
    return b["buckets"] if prev is None else (prev * b["mul_prev"] + cur * b["mul_cur"]) % b["buckets"]


def embedding(tokens: List[int], w: Dict[str, torch.Tensor], b: Optional[dict]):
    x = w["embed"][torch.tensor(tokens, dtype=torch.long)]
    if b:
        rows = [bigram_row(tokens[i - 1] if i else None, t, b) for i, t in enumerate(tokens)]
        x = x + w["bigram"][torch.tensor(rows, dtype=torch.long)]
    return x


# ------------------------------------------------------------------------------------------------ rotation
def scaled_frequency(f: float, s: dict) -> float:
    """A frequency under the three-zone scaling: short wavelengths stay, long ones are slowed by `factor`, a blend between."""
    length = 2.0 * math.pi / f
    if length < s["original"] / s["high"]:
        return f
    if length > s["original"] / s["low"]:
        return f / s["factor"]
    t = (s["original"] / length - s["low"]) / (s["high"] - s["low"])
    return (1.0 - t) * f / s["factor"] + t * f


def rotary_frequencies(dims: int, base: float, scaling: Optional[dict] = None) -> List[float]:
    """Angle per position step of pair i < dims / 2."""
    f = [base ** (-2.0 * i / dims) for i in range(dims // 2)]
    return [scaled_frequency(x, scaling) for x in f] if scaling else f


def rotate(x, rot: Optional[dict], positions=None):
    """x [T, ..., n], row t at position t (or positions[t]): entries i and i + dims / 2 of the first rot.dims turn by
    position * f_i, the rest pass."""
    y = x.clone()
    if not rot:
        return y
    dims = int(rot["dims"])
    pos = torch.arange(x.shape[0], dtype=F64) if positions is None else torch.as_tensor(positions, dtype=F64)
    pos = pos.view(-1, *([1] * (x.dim() - 2)))
    for i, f in enumerate(rotary_frequencies(dims, float(rot["base"]), rot.get("scaling"))):
        c, s = torch.cos(pos * f), torch.sin(pos * f)
        u, v = x[..., i], x[..., i + dims // 2]
        y[..., i] = u * c - v * s
        y[..., i + dims // 2] = v * c + u * s
    return y


# ------------------------------------------------------------------------------------------------ masks
def in_window(i: int, j: int, size: int) -> bool:
    """The query's own position and the size - 1 before it."""
    return 0 <= i - j < size


def in_window_or_kept(i: int, j: int, size: int, keep_first: int) -> bool:
    return j <= i and (i - j < size or j < keep_first)


def in_chunk(i: int, j: int, size: int) -> bool:
    """Causal inside blocks of `size` positions counted from the sequence's start."""
    return j <= i and i // size == j // size


def mask_matrix(T: int, seen: Callable[[int, int], bool]):
    return torch.tensor([[seen(i, j) for j in range(T)] for i in range(T)], dtype=torch.bool).view(T, T)


# ------------------------------------------------------------------------------------------------ attention
def softcap(s, cap: float):
    return cap * torch.tanh(s / cap)


def softmax_rows(scores, seen, sink: Optional[float] = None):
    """exp(s_j) / (sum over the keys seen + exp(sink)); sink None: no extra term."""
    s = torch.where(seen, scores, torch.full_like(scores, -math.inf))
    mx = s.max(dim=-1, keepdim=True).values
    if sink is not None:
        mx = torch.clamp(mx, min=sink)
    e = torch.exp(s - mx)
    den = e.sum(-1, keepdim=True)
    if sink is not None:
        den = den + torch.exp(sink - mx)
    return e / den


def attention(q, k, v, seen, scale: float, cap: Optional[float] = None, sinks=None):
    """q [T, H, dk], k [T, G, dk], v [T, G, dv], seen [T, T] -> [T, H, dv]; query head h reads key/value head h // (H / G)."""
    H, rep = q.shape[1], q.shape[1] // k.shape[1]
    out = []
    for h in range(H):
        s = q[:, h] @ k[:, h // rep].T * scale
        if cap:
            s = softcap(s, cap)
        out.append(softmax_rows(s, seen, None if sinks is None else float(sinks[h])) @ v[:, h // rep])
    return torch.stack(out, dim=1)


def diff_lambda(lq1, lk1, lq2, lk2, diff: float) -> float:
    return math.exp(float((lq1 * lk1).sum())) - math.exp(float((lq2 * lk2).sum())) + diff


def differential_attention(q, k, v, seen, scale: float, lam: float, diff: float, eps: float):
    """q [T, H, 2, dk], k [T, G, 2, dk], v [T, G, dv]: two softmax maps over the same values, the second subtracted lam times,
    the difference divided by its own root mean square and multiplied by 1 - diff."""
    a1 = attention(q[:, :, 0], k[:, :, 0], v, seen, scale)
    a2 = attention(q[:, :, 1], k[:, :, 1], v, seen, scale)
    return unit_rms(a1 - lam * a2, eps) * (1.0 - diff)


# ------------------------------------------------------------------------------------------------ retention
def retention(q, k, v, decay: List[float], S0=None):
    """q, k [T, H, dk], v [T, H, dv]: per head S <- decay S + k v^T, o = S^T q.  Returns o [T, H, dv] and the last S."""
    T, H, dk = q.shape
    S = torch.zeros(H, dk, v.shape[2], dtype=q.dtype) if S0 is None else S0.clone()
    d = torch.tensor(decay, dtype=q.dtype).view(H, 1, 1)
    out = []
    for t in range(T):
        S = d * S + k[t].unsqueeze(2) * v[t].unsqueeze(1)
        out.append((S * q[t].unsqueeze(2)).sum(1))
    return torch.stack(out), S


# ------------------------------------------------------------------------------------------------ mixers
def attention_mixer(h, w, p: str, m: dict, eps: float):
    """Windowed attention whose values are the keys as projected; q and k normed as whole rows, then rotated; capped scores and
    a sink per head."""
    T, H, G, dk = h.shape[0], m["heads"], m["kv_heads"], m["dim"]
    q = h @ w[p + ".q"].T + w[p + ".q.b"]
    k = h @ w[p + ".k"].T + w[p + ".k.b"]
    v = k.view(T, G, dk)
    q = rotate(rms_norm(q, w[p + ".q.norm"], eps).view(T, H, dk), m.get("rot"))
    k = rotate(rms_norm(k, w[p + ".k.norm"], eps).view(T, G, dk), m.get("rot"))
    seen = mask_matrix(T, lambda i, j: in_window(i, j, m["mask"]["size"]))
    o = attention(q, k, v, seen, m["scale"], m.get("softcap"), w[p + ".sink"])
    return o.reshape(T, H * dk) @ w[p + ".o"].T + w[p + ".o.b"]


def differential_mixer(h, w, p: str, m: dict, eps: float):
    T, H, G, dk, dv = h.shape[0], m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    q = rotate((h @ w[p + ".q"].T).view(T, H, 2, dk), m.get("rot"))
    k = rotate((h @ w[p + ".k"].T).view(T, G, 2, dk), m.get("rot"))
    v = (h @ w[p + ".v"].T).view(T, G, dv)
    lam = diff_lambda(w[p + ".lq1"], w[p + ".lk1"], w[p + ".lq2"], w[p + ".lk2"], m["diff"])
    seen = mask_matrix(T, lambda i, j: in_window_or_kept(i, j, m["mask"]["size"], m["mask"].get("keep_first", 0)))
    o = differential_attention(q, k, v, seen, m["scale"], lam, m["diff"], eps)
    return o.reshape(T, H * dv) @ w[p + ".o"].T


def chunk_mixer(h, w, p: str, m: dict, eps: float):
    T, H, G, dk, dv = h.shape[0], m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    q, k, v = (h @ w[f"{p}.{n}"].T + w[f"{p}.{n}.b"] for n in "qkv")
    q, k = rotate(q.view(T, H, dk), m.get("rot")), rotate(k.view(T, G, dk), m.get("rot"))
    seen = mask_matrix(T, lambda i, j: in_chunk(i, j, m["mask"]["size"]))
    o = attention(q, k, v.view(T, G, dv), seen, m["scale"])
    return o.reshape(T, H * dv) @ w[p + ".o"].T + w[p + ".o.b"]


def retention_mixer(h, w, p: str, m: dict, eps: float):
    T, H, dk, dv = h.shape[0], m["heads"], m["dim"], m["vdim"]
    q = rotate((h @ w[p + ".q"].T).view(T, H, dk), m.get("rot"))
    k = rotate((h @ w[p + ".k"].T).view(T, H, dk), m.get("rot")) * dk ** -0.5
    o, _ = retention(q, k, (h @ w[p + ".v"].T).view(T, H, dv), m["decay"])
    return (unit_rms(o, eps).reshape(T, H * dv) * silu(h @ w[p + ".g"].T)) @ w[p + ".o"].T


def parallel_mixer(h, w, p: str, m: dict, eps: float):
    left = rms_norm(chunk_mixer(h, w, p + ".left", m["left"], eps), w[p + ".left.out"], eps)
    right = rms_norm(retention_mixer(h, w, p + ".right", m["right"], eps), w[p + ".right.out"], eps)
    return 0.5 * (left + right)


MIXERS = {"attention": attention_mixer, "attention_2": differential_mixer, "parallel": parallel_mixer}


# ------------------------------------------------------------------------------------------------ feed-forward
def dense_ff(h, w, p: str, f: dict):
    return bounded_glu(h @ w[p + ".gate"].T, h @ w[p + ".up"].T, f["limit"]) @ w[p + ".down"].T


def expert(h, w, p: str):
    return (silu(h @ w[p + ".gate"].T) * (h @ w[p + ".up"].T)) @ w[p + ".down"].T


def route(h, w_router, top: int):
    """The `top` largest sigmoid scores per token and the scores themselves: ids, weights [T, top]."""
    s = sigmoid(h @ w_router.T)
    wts, ids = torch.topk(s, top, dim=-1)
    return ids, wts


def experts_ff(h, w, p: str, f: dict):
    """Sum over the chosen experts of expert(weight * h), plus the shared expert on h itself."""
    ids, wts = route(h, w[p + ".router"], f["router"]["top"])
    y = expert(h, w, p + ".shared") if f.get("shared") else torch.zeros_like(h)
    for t in range(h.shape[0]):
        for e, s in zip(ids[t].tolist(), wts[t]):
            y[t] = y[t] + expert(s * h[t], w, f"{p}.e{e}")
    return y


# ------------------------------------------------------------------------------------------------ the model
def _attention_shapes(q: str, m: dict, D: int) -> Dict[str, tuple]:
    return {q + ".q": (m["heads"] * m["dim"], D), q + ".k": (m["kv_heads"] * m["dim"], D)}


def tensor_shapes(cfg: dict) -> Dict[str, tuple]:
    """Name -> shape of a checkpoint's tensors."""
    D, V = cfg["width"], cfg["vocab"]
    out = {"embed": (V, D), "final.norm": (D,), "head": (V, D)}
    b = (cfg.get("embedding") or {}).get("bigram")
    if b:
        out["bigram"] = (b["buckets"] + 1, D)
    for i, L in enumerate(cfg["layers"]):
        p, m, f = f"l{i}", L["mixer"], L.get("mlp")
        q = p + ".mix"
        out.update({p + ".norm1": (D,), p + ".norm1b": (D,)})
        if L["type"] == "attention":
            out.update(_attention_shapes(q, m, D))
            nq, nk = m["heads"] * m["dim"], m["kv_heads"] * m["dim"]
            out.update({q + ".q.b": (nq,), q + ".k.b": (nk,), q + ".q.norm": (nq,), q + ".k.norm": (nk,),
                        q + ".sink": (m["heads"],), q + ".o": (D, nq), q + ".o.b": (D,)})
        elif L["type"] == "attention_2":
            out.update({q + ".q": (m["heads"] * 2 * m["dim"], D), q + ".k": (m["kv_heads"] * 2 * m["dim"], D),
                        q + ".v": (m["kv_heads"] * m["vdim"], D), q + ".o": (D, m["heads"] * m["vdim"])})
            out.update({f"{q}.{n}": (m["dim"],) for n in ("lq1", "lk1", "lq2", "lk2")})
        else:
            a, r, ql, qr = m["left"], m["right"], q + ".left", q + ".right"
            out.update(_attention_shapes(ql, a, D))
            out.update({ql + ".v": (a["kv_heads"] * a["vdim"], D), ql + ".q.b": (a["heads"] * a["dim"],),
                        ql + ".k.b": (a["kv_heads"] * a["dim"],), ql + ".v.b": (a["kv_heads"] * a["vdim"],),
                        ql + ".o": (D, a["heads"] * a["vdim"]), ql + ".o.b": (D,), ql + ".out": (D,)})
            nk, nv = r["heads"] * r["dim"], r["heads"] * r["vdim"]
            out.update({qr + ".q": (nk, D), qr + ".k": (nk, D), qr + ".v": (nv, D), qr + ".g": (nv, D), qr + ".o": (D, nv),
                        qr + ".out": (D,)})
        if not f:
            continue
        out.update({p + ".norm2": (D,), p + ".norm2b": (D,)})
        units = {"": f["ff"]} if f["kind"] == "dense" else {f".e{e}": f["expert"]["ff"] for e in range(f["router"]["experts"])}
        if f["kind"] == "moe":
            out[p + ".mlp.router"] = (f["router"]["experts"], D)
            if f.get("shared"):
                units[".shared"] = f["shared"]["ff"]
        for n, ff in units.items():
            out.update({f"{p}.mlp{n}.gate": (ff, D), f"{p}.mlp{n}.up": (ff, D), f"{p}.mlp{n}.down": (D, ff)})
    return out


def random_model(cfg: dict, seed: int = 0) -> Dict[str, torch.Tensor]:
    """Random bf16 tensors of a configuration: matrices with unit-variance outputs, norm weights around one, biases, sinks and
    lambda vectors of the order of what they sit beside."""
    g = torch.Generator().manual_seed(seed)
    out = {}
    for name, shape in tensor_shapes(cfg).items():
        t = torch.randn(*shape, generator=g, dtype=torch.float32)
        leaf = name.rsplit(".", 1)[-1]
        if leaf == "sink":
            t = 1.5 * t
        elif leaf == "b":
            t = 0.5 * t
        elif leaf in ("lq1", "lk1", "lq2", "lk2"):
            t = 0.6 * t * shape[0] ** -0.25
        elif leaf == "router":
            t = 2.0 * t * shape[-1] ** -0.5
        elif len(shape) == 1:
            t = 1.0 + 0.2 * t
        elif name not in ("embed", "bigram"):
            t = t * shape[-1] ** -0.5
        out[name] = t.to(torch.bfloat16)
    return out


def forward(cfg: dict, weights: Dict[str, torch.Tensor], tokens: List[int], layers_out: Optional[list] = None):
    """Logits [T, vocab] (float64) of one sequence from position 0; layers_out collects the residual after every layer."""
    w = {k: v.to(F64) for k, v in weights.items()}
    eps = float(cfg["norm"]["eps"])
    x = embedding(tokens, w, (cfg.get("embedding") or {}).get("bigram"))
    for i, L in enumerate(cfg["layers"]):
        p, f = f"l{i}", L.get("mlp")
        y = MIXERS[L["type"]](rms_norm(x, w[p + ".norm1"], eps), w, p + ".mix", L["mixer"], eps)
        x = x + rms_norm(y, w[p + ".norm1b"], eps)
        if f:
            h = rms_norm(x, w[p + ".norm2"], eps)
            y = dense_ff(h, w, p + ".mlp", f) if f["kind"] == "dense" else experts_ff(h, w, p + ".mlp", f)
            x = x + rms_norm(y, w[p + ".norm2b"], eps)
        if layers_out is not None:
            layers_out.append(x.clone())
    return rms_norm(x, w["final.norm"], eps) @ w["head"].T
