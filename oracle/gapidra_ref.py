"""Plain CPU restatement of the Gapidra decoder, one function per mechanism (test infrastructure only).

Everything runs in float64 on whole sequences; nothing here is shared with the product path under
vllm-backend-public_b200/ (which never imports this file).  `weights` maps the checkpoint's tensor names to tensors;
`cfg` is the parsed config.json dictionary.

Notation: T tokens, D model width, H query heads, G key/value heads, dk / dv per-head key and value sizes, dn / dr
per-head unrotated and rotated sizes of a latent layer, R latent size, W window.
"""
from __future__ import annotations

import math
from typing import Dict, List, Optional

import torch

F64 = torch.float64


# ------------------------------------------------------------------------------------------------ norm, activations
def rms_norm(x, w, eps):
    """x / sqrt(mean(x^2) + eps) * w over the last axis."""
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps) * w


def sigmoid(z):
    return 1.0 / (1.0 + torch.exp(-z))


def softplus(z: float) -> float:
    return math.log1p(math.exp(-abs(z))) + max(z, 0.0)


def xielu(z, p: float, q: float):
    """Quadratic above zero, exponential below, with the two curvatures learned: a = softplus(p), b = 1/2 + softplus(q);
    z > 0: a z^2 + z / 2;  z <= 0: b (e^z - 1 - z) + z / 2."""
    a, b = softplus(p), 0.5 + softplus(q)
    low = torch.clamp(z, max=0.0)
    return torch.where(z > 0, a * z * z, b * (torch.expm1(low) - low)) + 0.5 * z


# ------------------------------------------------------------------------------------------------ rotation
def yarn_ramp(dims: int, base: float, s: dict) -> List[float]:
    """Per pair i: 0 keeps the frequency, 1 divides it by s.factor.  The borders are the pairs that make `fast` and `slow`
    turns over the `original` positions."""
    def border(turns):
        return dims * math.log(s["original"] / (2.0 * math.pi * turns)) / (2.0 * math.log(base))
    lo = max(math.floor(border(s["fast"])), 0)
    hi = min(math.ceil(border(s["slow"])), dims - 1)
    return [min(max((i - lo) / max(hi - lo, 0.001), 0.0), 1.0) for i in range(dims // 2)]


def rotary_frequencies(dims: int, base: float, scaling: Optional[dict] = None) -> List[float]:
    """Angle per position step of pair i < dims / 2."""
    f = [base ** (-2.0 * i / dims) for i in range(dims // 2)]
    if scaling:
        f = [x / scaling["factor"] * r + x * (1.0 - r) for x, r in zip(f, yarn_ramp(dims, base, scaling))]
    return f


def rotary_magnitude(scaling: Optional[dict] = None) -> float:
    """Factor on cos and sin."""
    return 0.1 * math.log(scaling["factor"]) + 1.0 if scaling else 1.0


def rotate(x, rot: Optional[dict], layout: str):
    """x [T, ..., n], row t at position t: the first rot.dims entries turn by t * f_i per pair, the rest pass.  layout
    "half": entry i is paired with entry i + dims / 2; "interleaved": entry 2 i with entry 2 i + 1."""
    y = x.clone()
    if not rot:
        return y
    dims, scaling = int(rot["dims"]), rot.get("scaling")
    mag = rotary_magnitude(scaling)
    pos = torch.arange(x.shape[0], dtype=F64).view(-1, *([1] * (x.dim() - 2)))
    for i, f in enumerate(rotary_frequencies(dims, float(rot["base"]), scaling)):
        c, s = mag * torch.cos(pos * f), mag * torch.sin(pos * f)
        p, q = (i, i + dims // 2) if layout == "half" else (2 * i, 2 * i + 1)
        u, v = x[..., p], x[..., q]
        y[..., p] = u * c - v * s
        y[..., q] = v * c + u * s
    return y


# ------------------------------------------------------------------------------------------------ masks and weights
def visible(i: int, j: int, window: int) -> bool:
    """Whether the query at position i sees the key at position j: causal; with a window (> 0) only the last `window`
    positions, its own included."""
    return j <= i and (window <= 0 or i - j < window)


def mask_matrix(T: int, window: int):
    return torch.tensor([[visible(i, j, window) for j in range(T)] for i in range(T)], dtype=torch.bool)


def sink_softmax(scores, seen, sink: Optional[float]):
    """Rows of scores [T, T] under the mask `seen`: exp(s_j) / (sum_j exp(s_j) + exp(sink)); sink None: no extra term."""
    s = torch.where(seen, scores, torch.full_like(scores, -math.inf))
    mx = s.max(dim=-1, keepdim=True).values
    if sink is not None:
        mx = torch.clamp(mx, min=sink)
    e = torch.exp(s - mx)
    den = e.sum(-1, keepdim=True)
    if sink is not None:
        den = den + torch.exp(sink - mx)
    return e / den


def sigmoid_weights(scores, seen, bias: float):
    """sigmoid(s_j + bias) for the keys seen, 0 elsewhere; a key's weight does not depend on the other keys."""
    return torch.where(seen, sigmoid(scores + bias), torch.zeros_like(scores))


def softmax_attention(q, k, v, scale: float, window: int = 0, sinks=None):
    """q [T, H, dk], k [T, G, dk], v [T, G, dv] -> [T, H, dv]; query head h reads key/value head h // (H / G)."""
    T, H, _ = q.shape
    seen, rep = mask_matrix(T, window), H // k.shape[1]
    return torch.stack([sink_softmax(q[:, h] @ k[:, h // rep].T * scale, seen, None if sinks is None else float(sinks[h]))
                        @ v[:, h // rep] for h in range(H)], dim=1)


def sigmoid_attention(q, k, v, scale: float, window: int, bias):
    """The same with sigmoid weights, bias [H]."""
    T, H, _ = q.shape
    seen, rep = mask_matrix(T, window), H // k.shape[1]
    return torch.stack([sigmoid_weights(q[:, h] @ k[:, h // rep].T * scale, seen, float(bias[h])) @ v[:, h // rep]
                        for h in range(H)], dim=1)


# ------------------------------------------------------------------------------------------------ mixers
def window_of(m: dict) -> int:
    return int((m.get("mask") or {}).get("size") or 0)


def latent_keys_values(c, kt, w_uk, w_uv, H: int):
    """Per head keys [T, H, dn + dr] = [W_uk c | shared rotated part] and values [T, H, dv] = W_uv c."""
    T = c.shape[0]
    kn = (c @ w_uk.T).view(T, H, -1)
    return torch.cat([kn, kt.unsqueeze(1).expand(T, H, kt.shape[1])], dim=-1), (c @ w_uv.T).view(T, H, -1)


def latent_mixer(h, w: Dict[str, torch.Tensor], p: str, m: dict, eps: float):
    """Windowed softmax attention with a sink per head over a shared latent, gated per channel.  h [T, D] -> [T, D]."""
    T = h.shape[0]
    H, dn, dr, dv, R = m["heads"], m["dim"], m["rot_dim"], m["vdim"], m["kv_rank"]
    q = (h @ w[p + ".q"].T).view(T, H, dn + dr)
    dkv = h @ w[p + ".dkv"].T
    c = rms_norm(dkv[:, :R], w[p + ".dkv.norm"], eps)
    kt = rotate(dkv[:, R:], m.get("rot"), "half")
    q = torch.cat([q[..., :dn], rotate(q[..., dn:], m.get("rot"), "half")], dim=-1)
    k, v = latent_keys_values(c, kt, w[p + ".uk"], w[p + ".uv"], H)
    o = softmax_attention(q, k, v, m["scale"], window_of(m), w[p + ".sink"]).reshape(T, H * dv)
    return (o * sigmoid(h @ w[p + ".g"].T)) @ w[p + ".o"].T


def sigmoid_mixer(h, w: Dict[str, torch.Tensor], p: str, m: dict, eps: float):
    """Windowed grouped-query attention with sigmoid weights; q and k normed over the whole projection, then rotated.
    h [T, D] -> [T, D]."""
    T = h.shape[0]
    H, G = m["heads"], m["kv_heads"]
    q = rms_norm(h @ w[p + ".q"].T, w[p + ".q.norm"], eps).view(T, H, m["dim"])
    k = rms_norm(h @ w[p + ".k"].T, w[p + ".k.norm"], eps).view(T, G, m["dim"])
    v = (h @ w[p + ".v"].T).view(T, G, m["vdim"])
    q, k = rotate(q, m.get("rot"), "interleaved"), rotate(k, m.get("rot"), "interleaved")
    o = sigmoid_attention(q, k, v, m["scale"], window_of(m), w[p + ".pb"])
    return o.reshape(T, H * m["vdim"]) @ w[p + ".o"].T


def dense_ff(h, w: Dict[str, torch.Tensor], p: str):
    """W_down xielu(W_up h)."""
    a = w[p + ".act"]
    return xielu(h @ w[p + ".up"].T, float(a[0]), float(a[1])) @ w[p + ".down"].T


# ------------------------------------------------------------------------------------------------ the model
def tensor_shapes(cfg: dict) -> Dict[str, tuple]:
    """Name -> shape of a checkpoint's tensors."""
    D, V = cfg["width"], cfg["vocab"]
    out = {"embed": (V, D), "final.norm": (D,), "head": (V, D)}
    for i, L in enumerate(cfg["layers"]):
        p, m = f"l{i}", L["mixer"]
        q, H = p + ".mix", m["heads"]
        out[p + ".norm1"] = (D,)
        if L["type"] == "latent_attention":
            R = m["kv_rank"]
            out.update({q + ".q": (H * (m["dim"] + m["rot_dim"]), D), q + ".dkv": (R + m["rot_dim"], D), q + ".dkv.norm": (R,),
                        q + ".uk": (H * m["dim"], R), q + ".uv": (H * m["vdim"], R), q + ".sink": (H,),
                        q + ".g": (H * m["vdim"], D)})
        else:
            G = m["kv_heads"]
            out.update({q + ".q": (H * m["dim"], D), q + ".k": (G * m["dim"], D), q + ".v": (G * m["vdim"], D),
                        q + ".q.norm": (H * m["dim"],), q + ".k.norm": (G * m["dim"],), q + ".pb": (H,)})
        out[q + ".o"] = (D, H * m["vdim"])
        if L.get("mlp"):
            out.update({p + ".mlp.up": (L["mlp"]["ff"], D), p + ".mlp.down": (D, L["mlp"]["ff"]), p + ".mlp.act": (2,)})
    return out


def random_model(cfg: dict, seed: int = 0) -> Dict[str, torch.Tensor]:
    """Random bf16 tensors of a configuration: matrices with unit-variance outputs, norm weights around one, sinks, score
    biases and activation numbers of the order of what they sit beside."""
    g = torch.Generator().manual_seed(seed)
    out = {}
    for name, shape in tensor_shapes(cfg).items():
        t = torch.randn(*shape, generator=g, dtype=torch.float32)
        if name.endswith(".sink"):
            t = 1.5 * t
        elif name.endswith(".pb"):
            t = t - 2.0
        elif name.endswith(".act"):
            t = 0.7 * t
        elif len(shape) == 1:
            t = 1.0 + 0.2 * t
        elif name != "embed":
            t = t * shape[-1] ** -0.5
        out[name] = t.to(torch.bfloat16)
    return out


def forward(cfg: dict, weights: Dict[str, torch.Tensor], tokens: List[int], layers_out: Optional[list] = None):
    """Logits [T, vocab] (float64) of one sequence from position 0; layers_out collects the residual after every layer."""
    w = {k: v.to(F64) for k, v in weights.items()}
    eps = float(cfg["norm"]["eps"])
    x = w["embed"][torch.tensor(tokens, dtype=torch.long)] * float(cfg["embedding"]["scale"])
    for i, L in enumerate(cfg["layers"]):
        p = f"l{i}"
        h = rms_norm(x, w[p + ".norm1"], eps)
        if L["type"] == "latent_attention":
            y = latent_mixer(h, w, p + ".mix", L["mixer"], eps)
        elif L["type"] == "attention":
            y = sigmoid_mixer(h, w, p + ".mix", L["mixer"], eps)
        else:
            raise ValueError(f"layer {i}: unknown mixer {L['type']!r}")
        if L.get("mlp"):
            if L["mlp"]["kind"] != "dense":
                raise ValueError(f"layer {i}: unknown feed-forward {L['mlp']['kind']!r}")
            y = y + dense_ff(h, w, p + ".mlp")           # both sublayers read the same norm's output
        x = x + y
        if layers_out is not None:
            layers_out.append(x.clone())
    return rms_norm(x, w["final.norm"], eps) @ w["head"].T
