"""Lizazen decoder on the b200attn ops: RMS norms before AND after every sublayer around one fp32 residual, an embedding that adds
a hashed bigram row (the token before is per-sequence state), and one of three sequence mixers per layer:

  attention     sliding-window grouped-query softmax attention whose values are the keys as projected; q and k are RMS-normed
                over the whole projection, then partly rotated (pairs (i, i + dims/2), three-zone frequency scaling); scores are
                soft-capped and a learned sink per head joins the denominator.
  attention_2   differential attention: every head holds two softmax maps over the same values, the second is subtracted lambda
                times and the difference normed per head; sliding window that keeps the sequence's first tokens.
  parallel      two mixers that read the same input, each output RMS-normed over the width, half their sum: chunk-masked softmax
                attention with biased projections, and retention (linear attention with a fixed decay per head over rotated q and
                k, a norm per head, SiLU gate) whose matrix state lives in fp32 state slots.

The feed-forward is dense with bounded gated units, a routed mixture of SiLU-gated experts whose sigmoid scores weight the
experts' INPUT beside a shared expert, or absent.

The model plugs into the same engine as the other families (b200attn.engine.LLMEngine): paged pools addressed through the
scheduler's block tables and slot mapping, state slots per live sequence, one forward over [decode rows | prompt chunks],
logits for the sampled rows.  Projections and the vocabulary head are library GEMMs (torch -> cuBLAS); everything between
them is this repo's kernels (csrc/hyper_norm.cu, post_norm.cu, chunk_attention.cu, delta_rule.cu, moe.cu).  There is no CPU
path.

Every size, the layer order and every constant come from the checkpoint's config.json (`architecture: "Lizazen"`);
weights from its *.safetensors, or random from a seed.
"""
from __future__ import annotations

import json
import math
import os
from dataclasses import dataclass
from pathlib import Path
from typing import Dict, List, Optional, Tuple, Union

import torch

from . import ops

ARCHITECTURE = "Lizazen"
GLU_ALPHA = 1.702            # the design fixes the slope of the bounded units' sigmoid
PAIR_SCALE = 0.5             # ... and the weight of the two halves of a parallel mixer
LAMBDA_VECTORS = ("lq1", "lk1", "lq2", "lk2")


@dataclass(frozen=True)
class Rotation:
    dims: int = 0              # how many leading entries turn (the rest pass)
    base: float = 10000.0
    scaling: Optional[Tuple[Tuple[str, float], ...]] = None     # sorted items of {factor, low, high, original}


@dataclass(frozen=True)
class WindowSpec:
    heads: int
    kv_heads: int
    dim: int                   # per-head query / key size; the values are the keys, so also the value size
    scale: float
    softcap: float             # 0: the scores are not capped
    window: int                # a query sees its own position and the window - 1 before it (0: plain causal)
    rot: Rotation


@dataclass(frozen=True)
class DiffSpec:
    heads: int
    kv_heads: int
    dim: int                   # query / key size of ONE map; a head holds two
    vdim: int
    scale: float
    diff: float
    window: int
    keep_first: int            # ... and the first keep_first positions of the sequence
    rot: Rotation


@dataclass(frozen=True)
class ChunkSpec:
    heads: int
    kv_heads: int
    dim: int
    vdim: int
    scale: float
    chunk: int                 # a query sees the keys of its own block of this many positions (0: plain causal)
    rot: Rotation


@dataclass(frozen=True)
class RetentionSpec:
    heads: int
    dim: int
    vdim: int
    decay: Tuple[float, ...]   # one fixed factor per head
    rot: Rotation


@dataclass(frozen=True)
class ParallelSpec:
    left: ChunkSpec
    right: RetentionSpec


@dataclass(frozen=True)
class DenseSpec:
    ff: int
    limit: float


@dataclass(frozen=True)
class ExpertsSpec:
    experts: int
    top: int
    ff: int
    shared_ff: int             # 0: no shared expert


MixerSpec = Union[WindowSpec, DiffSpec, ParallelSpec]


@dataclass(frozen=True)
class LayerSpec:
    mixer: MixerSpec
    mlp: Union[None, DenseSpec, ExpertsSpec]


def _pad8(n: int) -> int:
    return (n + 7) // 8 * 8


def _attention_of(m: MixerSpec) -> Union[WindowSpec, DiffSpec, ChunkSpec]:
    """The part of a mixer that keeps keys and values."""
    return m.left if isinstance(m, ParallelSpec) else m


def _pool_heads(m: MixerSpec) -> Tuple[int, int, int, int]:
    """(key heads, key size, value heads, value size) of a layer's pools."""
    a = _attention_of(m)
    if isinstance(a, DiffSpec):
        return 2 * a.kv_heads, a.dim, a.kv_heads, a.vdim
    return a.kv_heads, a.dim, a.kv_heads, a.dim if isinstance(a, WindowSpec) else a.vdim


def layer_tensors(p: str, L: LayerSpec, D: int) -> Dict[str, Tuple[int, ...]]:
    """Name -> shape of one layer's tensors."""
    m, f, q = L.mixer, L.mlp, p + ".mix"
    out: Dict[str, Tuple[int, ...]] = {p + ".norm1": (D,), p + ".norm1b": (D,)}
    if isinstance(m, WindowSpec):
        nq, nk = m.heads * m.dim, m.kv_heads * m.dim
        out.update({q + ".q": (nq, D), q + ".q.b": (nq,), q + ".k": (nk, D), q + ".k.b": (nk,), q + ".q.norm": (nq,),
                    q + ".k.norm": (nk,), q + ".sink": (m.heads,), q + ".o": (D, nq), q + ".o.b": (D,)})
    elif isinstance(m, DiffSpec):
        out.update({q + ".q": (2 * m.heads * m.dim, D), q + ".k": (2 * m.kv_heads * m.dim, D), q + ".v": (m.kv_heads * m.vdim, D),
                    q + ".o": (D, m.heads * m.vdim)})
        out.update({f"{q}.{n}": (m.dim,) for n in LAMBDA_VECTORS})
    else:
        a, r, ql, qr = m.left, m.right, q + ".left", q + ".right"
        for n, rows in (("q", a.heads * a.dim), ("k", a.kv_heads * a.dim), ("v", a.kv_heads * a.vdim)):
            out.update({f"{ql}.{n}": (rows, D), f"{ql}.{n}.b": (rows,)})
        out.update({ql + ".o": (D, a.heads * a.vdim), ql + ".o.b": (D,), ql + ".out": (D,)})
        for n, rows in (("q", r.heads * r.dim), ("k", r.heads * r.dim), ("v", r.heads * r.vdim), ("g", r.heads * r.vdim)):
            out[f"{qr}.{n}"] = (rows, D)
        out.update({qr + ".o": (D, r.heads * r.vdim), qr + ".out": (D,)})
    if f is None:
        return out
    out.update({p + ".norm2": (D,), p + ".norm2b": (D,)})
    units = {"": f.ff} if isinstance(f, DenseSpec) else {f".e{e}": f.ff for e in range(f.experts)}
    if isinstance(f, ExpertsSpec):
        out[p + ".mlp.router"] = (f.experts, D)
        if f.shared_ff:
            units[".shared"] = f.shared_ff
    for n, ff in units.items():
        out.update({f"{p}.mlp{n}.gate": (ff, D), f"{p}.mlp{n}.up": (ff, D), f"{p}.mlp{n}.down": (D, ff)})
    return out


@dataclass
class LizazenConfig:
    name: str
    vocab: int
    hidden: int
    layer_specs: List[LayerSpec]
    eps: float = 1e-6
    buckets: int = 0                       # rows of the bigram table less one (0: no bigram embedding)
    mul_prev: int = 0
    mul_cur: int = 0
    max_position: int = 1 << 20            # the rotary tables are built for the engine's max_model_len
    family: str = "lizazen"

    @property
    def layers(self) -> int:
        return len(self.layer_specs)

    def tensors(self) -> Dict[str, Tuple[int, ...]]:
        """Name -> shape of every tensor of a checkpoint of this configuration."""
        D = self.hidden
        out: Dict[str, Tuple[int, ...]] = {"embed": (self.vocab, D), "final.norm": (D,), "head": (self.vocab, D)}
        if self.buckets:
            out["bigram"] = (self.buckets + 1, D)
        for i, L in enumerate(self.layer_specs):
            out.update(layer_tensors(f"l{i}", L, D))
        return out

    @property
    def params(self) -> int:
        return sum(math.prod(s) for s in self.tensors().values())

    def kv_bytes_per_token(self, kv_elem_bytes: int = 2, tp: int = 1) -> int:
        n = 0
        for L in self.layer_specs:
            gk, dk, gv, dv = _pool_heads(L.mixer)
            n += (gk * dk + gv * dv) * kv_elem_bytes
        return n

    def state_bytes_per_seq(self, elem_bytes: int = 2) -> int:
        """The fp32 matrix state of every parallel layer, and the token before."""
        rs = [L.mixer.right for L in self.layer_specs if isinstance(L.mixer, ParallelSpec)]
        return sum(r.heads * r.dim * r.vdim * 4 for r in rs) + 8

    def activation_bytes(self, tokens: int, seqs: int, elem_bytes: int = 2) -> int:
        wide, moe = [self.hidden], [0]
        for L in self.layer_specs:
            m, f = L.mixer, L.mlp
            a = _attention_of(m)
            gk, dk, gv, dv = _pool_heads(m)
            n = 2 * a.heads * (gk // gv) * dk + gk * dk + gv * dv + a.heads * dv
            if isinstance(m, ParallelSpec):            # the retention's rows also exist in fp32
                n += 3 * m.right.heads * (2 * m.right.dim + 3 * m.right.vdim) + 2 * self.hidden
            if isinstance(f, DenseSpec):
                n = max(n, 3 * f.ff)
            elif f is not None:
                n = max(n, 3 * f.shared_ff)
                moe.append(f.top * (3 * f.ff * elem_bytes + self.hidden * 4))
            wide.append(n)
        return tokens * (self.hidden * 12 + 2 * max(wide) * elem_bytes + 2 * max(moe)) + seqs * self.vocab * 8 + (1 << 28)

    def build_model(self, device, **kw):
        return LizazenModel(self, device, **kw)


def _rotation(m: dict, where: str) -> Rotation:
    rot = m.get("rot")
    if not rot:
        return Rotation()
    s = rot.get("scaling")
    r = Rotation(int(rot.get("dims", m["dim"])), float(rot.get("base", 10000.0)),
                 tuple(sorted((k, float(v)) for k, v in s.items())) if s else None)
    if r.dims % 2 or not 0 <= r.dims <= int(m["dim"]):
        raise ValueError(f"{where}: rot.dims {r.dims} must be even and at most dim {m['dim']}")
    if s and not {"factor", "low", "high", "original"} <= set(s):
        raise ValueError(f"{where}: rot.scaling needs factor, low, high and original")
    if s and not float(s["low"]) < float(s["high"]):
        raise ValueError(f"{where}: rot.scaling.low must be below high")
    return r


def _heads(m: dict, where: str) -> Tuple[int, int]:
    h, g = int(m["heads"]), int(m.get("kv_heads", m["heads"]))
    if g < 1 or h % g:
        raise ValueError(f"{where}: {h} query heads over {g} key/value heads")
    return h, g


def _mask(m: dict, key: str, where: str) -> int:
    v = int((m.get("mask") or {}).get(key) or 0)
    if v < 0:
        raise ValueError(f"{where}: mask.{key} {v} is negative")
    return v


def _mixer(kind: str, m: dict, where: str) -> MixerSpec:
    if kind == "attention":
        h, g = _heads(m, where)
        if int(m.get("vdim", m["dim"])) != int(m["dim"]):
            raise ValueError(f"{where}: the values are the keys, vdim {m['vdim']} must equal dim {m['dim']}")
        cap = float(m.get("softcap") or 0.0)
        if cap < 0:
            raise ValueError(f"{where}: softcap {cap} is negative")
        return WindowSpec(h, g, int(m["dim"]), float(m["scale"]), cap, _mask(m, "size", where), _rotation(m, where))
    if kind == "attention_2":
        h, g = _heads(m, where)
        return DiffSpec(h, g, int(m["dim"]), int(m.get("vdim", m["dim"])), float(m["scale"]), float(m["diff"]), _mask(m, "size", where),
                        _mask(m, "keep_first", where), _rotation(m, where))
    if kind == "parallel":
        a, r = m["left"], m["right"]
        h, g = _heads(a, where + " left")
        left = ChunkSpec(h, g, int(a["dim"]), int(a.get("vdim", a["dim"])), float(a["scale"]), _mask(a, "size", where), _rotation(a, where))
        right = RetentionSpec(int(r["heads"]), int(r["dim"]), int(r.get("vdim", r["dim"])), tuple(float(x) for x in r["decay"]),
                              _rotation(r, where))
        if len(right.decay) != right.heads:
            raise ValueError(f"{where}: {len(right.decay)} decay factors for {right.heads} heads")
        return ParallelSpec(left, right)
    raise ValueError(f"{where}: unknown mixer type {kind!r}")


def _feed_forward(f: Optional[dict], where: str) -> Union[None, DenseSpec, ExpertsSpec]:
    if not f:
        return None
    if f.get("kind") == "dense":
        return DenseSpec(int(f["ff"]), float(f["limit"]))
    if f.get("kind") == "moe":
        r = f["router"]
        e = ExpertsSpec(int(r["experts"]), int(r["top"]), int(f["expert"]["ff"]), int((f.get("shared") or {}).get("ff", 0)))
        if not 1 <= e.top <= e.experts:
            raise ValueError(f"{where}: router picks {e.top} of {e.experts} experts")
        return e
    raise ValueError(f"{where}: unknown feed-forward kind {f.get('kind')!r}")


def config_from_dict(c: dict, name: str = ARCHITECTURE) -> LizazenConfig:
    """config.json -> LizazenConfig.  Keys: vocab, width, norm.eps, embedding.bigram {buckets, mul_prev, mul_cur}, layers [{type,
    mixer, mlp null | {kind: dense, ff, limit} | {kind: moe, expert {ff}, router {experts, top}, shared null | {ff}}}] with the
    mixers
      attention    {heads, kv_heads, dim, vdim (= dim), scale, softcap, mask {size}, rot {base, dims, scaling {factor, low, high, original}}}
      attention_2  {heads, kv_heads, dim, vdim, scale, diff, mask {size, keep_first}, rot}
      parallel     {left {heads, kv_heads, dim, vdim, scale, mask {size}, rot}, right {heads, dim, vdim, decay [heads], rot}}."""
    specs = [LayerSpec(_mixer(L["type"], L["mixer"], f"layer {i}"), _feed_forward(L.get("mlp"), f"layer {i}"))
             for i, L in enumerate(c["layers"])]
    b = (c.get("embedding") or {}).get("bigram") or {}
    out = LizazenConfig(name=name, vocab=int(c["vocab"]), hidden=int(c["width"]), layer_specs=specs,
                        eps=float((c.get("norm") or {}).get("eps", 1e-6)), buckets=int(b.get("buckets", 0)),
                        mul_prev=int(b.get("mul_prev", 0)), mul_cur=int(b.get("mul_cur", 0)))
    if b and (out.buckets < 1 or out.mul_prev < 0 or out.mul_cur < 0):
        raise ValueError("embedding.bigram needs at least one bucket and multipliers that are not negative")
    return out


def config_from_dir(path: Path) -> LizazenConfig:
    path = Path(path)
    return config_from_dict(json.loads((path / "config.json").read_text()), name=path.name)


def bench_config(hidden: int, layers: int, heads: int, kv_heads: int, head_dim: int, ff: int, experts: int, top: int, vocab: int,
                 window: int = 1024, keep_first: int = 4, chunk: int = 1024, buckets: int = 65521,
                 name: str = "lizazen-bench") -> LizazenConfig:
    """A model-sized geometry for benchmarks: attention, attention_2 and parallel layers in turn (the maps of a differential head
    hold half a head's size each); the attention layers carry a dense feed-forward of the experts' active width, the others
    routed experts, one of the chosen width shared."""
    zones = (("factor", 8.0), ("high", 4.0), ("low", 1.0), ("original", 8192.0))
    specs = []
    for i in range(layers):
        kind = i % 3
        if kind == 0:
            m: MixerSpec = WindowSpec(heads, kv_heads, head_dim, head_dim ** -0.5, 50.0, window, Rotation(head_dim, 5e5, zones))
        elif kind == 1:
            m = DiffSpec(heads, kv_heads, head_dim // 2, head_dim, (head_dim // 2) ** -0.5, 0.4, window, keep_first,
                         Rotation(head_dim // 2, 1e6))
        else:
            n = max(heads // 2, 1)
            decay = tuple(1.0 - 2.0 ** (-5.0 - 3.0 * h / max(n - 1, 1)) for h in range(n))
            m = ParallelSpec(ChunkSpec(heads, kv_heads, head_dim, head_dim, head_dim ** -0.5, chunk, Rotation(head_dim // 2, 1e6)),
                             RetentionSpec(n, head_dim, head_dim, decay, Rotation(head_dim, 1e4)))
        specs.append(LayerSpec(m, DenseSpec(ff * top, 7.0) if kind == 0 else ExpertsSpec(experts, max(top - 1, 1), ff, ff)))
    return LizazenConfig(name, vocab, hidden, specs, buckets=buckets, mul_prev=1009, mul_cur=31)


class LizazenModel:
    """Weights + per-layer pools and states + forward over one scheduled token batch.  One instance per GPU."""

    supports_fp32 = True
    launches_per_layer = 10

    def __init__(self, cfg: LizazenConfig, device: torch.device, num_blocks: int, block_size: int = 16, seed: int = 0,
                 weights_dir: Optional[Path] = None, max_position: Optional[int] = None,
                 kv_dtype: torch.dtype = torch.bfloat16, tp=None, dtype: torch.dtype = torch.bfloat16,
                 max_num_seqs: int = 1):
        if device.type != "cuda":
            raise ValueError("LizazenModel needs a CUDA device (b200attn has no CPU path)")
        if tp is not None and tp.size > 1:
            raise ValueError("Lizazen runs on one GPU per replica: tensor_parallel_size must be 1")
        if dtype not in (torch.bfloat16, torch.float32):
            raise ValueError(f"dtype {dtype}: bfloat16 or float32")
        if kv_dtype not in (torch.bfloat16, dtype):
            raise ValueError("Lizazen keeps its pools in the activation type (no fp8 cache)")
        self.cfg, self.dev, self.bs, self.dtype = cfg, device, block_size, dtype
        self.tp, self.tp_size, self.tp_rank = None, 1, 0
        self.vocab_parallel = False
        self.Hq = self.Hkv = 0                      # no paged-decode schedule to plan
        self.max_position = max_position or min(cfg.max_position, 1 << 17)
        self.max_num_seqs = max_num_seqs
        self.w: Dict[str, torch.Tensor] = {}
        self.cols: Dict[int, Dict[str, int]] = {}   # layer -> first column of every part of its fused projection
        self.lam: Dict[int, float] = {}             # differential layer -> the weight of its second map
        if weights_dir is not None and any(Path(weights_dir).glob("*.safetensors")):
            self._load(Path(weights_dir))
        else:
            self._random_init(seed)
        self._fuse()
        # one rotary table per distinct (dims, base, scaling)
        self.rot: Dict[Rotation, Optional[torch.Tensor]] = {}
        for L in cfg.layer_specs:
            m = L.mixer
            for r in (m.left.rot, m.right.rot) if isinstance(m, ParallelSpec) else (m.rot,):
                if r not in self.rot:
                    self.rot[r] = ops.rotary_table(self.max_position, r.dims, r.base, dict(r.scaling) if r.scaling else None, device) \
                        if r.dims else None
        self.num_blocks = 0
        self.k_cache: Dict[int, torch.Tensor] = {}
        self.v_cache: Dict[int, torch.Tensor] = {}
        self.state: Dict[int, torch.Tensor] = {}
        self.last_token: Optional[torch.Tensor] = None
        self.alloc_cache(num_blocks)
        self.alloc_state(max_num_seqs)
        self._arange = torch.arange(max_num_seqs + 1, dtype=torch.int32, device=device)
        # the two halves of a parallel mixer are independent between the fused projection and the norm of their sum: the
        # recurrent half (few CTAs, a dependent chain per sequence) runs on a second stream under the attention
        self.overlap = os.environ.get("B2_PARALLEL_MIXER_STREAMS", "1") != "0"
        self._side = torch.cuda.Stream(device)
        self.capture: Optional[list] = None         # tests: set to a list to collect the residual after every layer

    # ------------------------------------------------------------------ weights
    def _random_init(self, seed: int) -> None:
        g = torch.Generator(device=self.dev).manual_seed(seed)
        raw = {}
        for name, shape in self.cfg.tensors().items():
            leaf = name.rsplit(".", 1)[-1]
            t = torch.randn(*shape, generator=g, device=self.dev, dtype=torch.float32)
            if leaf in LAMBDA_VECTORS or leaf == "b":
                t = 0.1 * t
            elif len(shape) == 1 and leaf != "sink":
                t = 1.0 + 0.1 * t
            elif len(shape) == 2 and name not in ("embed", "bigram"):
                t = t * shape[-1] ** -0.5
            raw[name] = t.to(torch.bfloat16)
        self._ingest(raw)

    def _load(self, path: Path) -> None:
        from safetensors import safe_open
        raw: Dict[str, torch.Tensor] = {}
        for f in sorted(path.glob("*.safetensors")):
            with safe_open(str(f), framework="pt", device="cpu") as sf:
                for k in sf.keys():
                    raw[k] = sf.get_tensor(k)
        want = self.cfg.tensors()
        missing = [k for k in want if k not in raw]
        if missing:
            raise ValueError(f"checkpoint lacks {len(missing)} tensors, e.g. {missing[:3]}")
        for k, shape in want.items():
            if tuple(raw[k].shape) != tuple(shape):
                raise ValueError(f"{k}: shape {tuple(raw[k].shape)} in the checkpoint, {tuple(shape)} by config.json")
        self._ingest({k: raw[k].to(self.dev) for k in want})

    def _ingest(self, raw: Dict[str, torch.Tensor]) -> None:
        """Matrices and projection biases in the activation type, parameter vectors in fp32."""
        for k, t in raw.items():
            self.w[k] = t.to(torch.float32 if t.dim() == 1 and not k.endswith(".b") else self.dtype).contiguous()

    def _stack(self, li: int, parts: List[Tuple[str, List[str]]]) -> torch.Tensor:
        """Rows of several matrices as one projection matrix; every named part starts on a multiple of eight rows (zero rows
        between), so that the columns it produces stay 16-byte aligned.  Records the parts' first columns; takes the matrices
        out of self.w, and their biases, if any has one, into one bias vector of the fused product."""
        rows, bias, cols, at = [], [], {}, 0
        biased = any(n + ".b" in self.w for _, names in parts for n in names)
        for name, names in parts:
            cols[name] = at
            for n in names:
                m = self.w.pop(n)
                rows.append(m)
                bias.append(self.w.pop(n + ".b", None))
                if bias[-1] is None:
                    bias[-1] = torch.zeros(m.shape[0], dtype=self.dtype, device=self.dev)
                at += m.shape[0]
            pad = -at % 8
            if pad:
                rows.append(torch.zeros(pad, rows[0].shape[1], dtype=self.dtype, device=self.dev))
                bias.append(torch.zeros(pad, dtype=self.dtype, device=self.dev))
            at += pad
        self.cols[li] = cols
        if biased:
            self.w[f"l{li}.bproj"] = torch.cat(bias).contiguous()
        return torch.cat(rows).contiguous()

    def _fuse(self) -> None:
        """Per layer: ONE projection matrix for everything that reads the mixer's input (with the biases as one vector), gate and
        up stacked (dense units, the shared expert, and per expert), the number a differential layer subtracts by."""
        w, c = self.w, self.cfg
        pop = w.pop
        for i, L in enumerate(c.layer_specs):
            p, m, f, q = f"l{i}", L.mixer, L.mlp, f"l{i}.mix"
            if isinstance(m, WindowSpec):
                parts = [("qk", [q + ".q", q + ".k"])]
            elif isinstance(m, DiffSpec):
                parts = [("qkv", [q + ".q", q + ".k", q + ".v"])]
                lq1, lk1, lq2, lk2 = (pop(f"{q}.{n}").double() for n in LAMBDA_VECTORS)
                self.lam[i] = math.exp(float((lq1 * lk1).sum())) - math.exp(float((lq2 * lk2).sum())) + m.diff
            else:
                ql, qr = q + ".left", q + ".right"
                parts = [("left", [ql + ".q", ql + ".k", ql + ".v"]), ("right", [qr + ".q", qr + ".k", qr + ".v"]), ("g", [qr + ".g"])]
                w[qr + ".decay"] = torch.tensor(m.right.decay, dtype=torch.float32, device=self.dev)
            w[p + ".wproj"] = self._stack(i, parts)
            u = p + ".mlp"
            if isinstance(f, DenseSpec):
                w[u + ".gate_up"] = torch.cat([pop(u + ".gate"), pop(u + ".up")]).contiguous()
            elif f is not None:
                w[u + ".gate_up"] = torch.stack([torch.cat([pop(f"{u}.e{e}.gate"), pop(f"{u}.e{e}.up")]) for e in range(f.experts)]).contiguous()
                w[u + ".down"] = torch.stack([pop(f"{u}.e{e}.down") for e in range(f.experts)]).contiguous()
                if f.shared_ff:
                    w[u + ".shared.gate_up"] = torch.cat([pop(u + ".shared.gate"), pop(u + ".shared.up")]).contiguous()

    def weight_bytes(self) -> int:
        return sum(t.numel() * t.element_size() for t in self.w.values())

    # ------------------------------------------------------------------ caches and state
    def alloc_cache(self, num_blocks: int) -> None:
        """Per layer a K pool (rotated keys) [num_blocks, key heads, bs, dim] and a V pool [num_blocks, value heads, bs, vdim]; a
        differential layer has two key heads (its maps) for every value head."""
        self.num_blocks = int(num_blocks)
        self.k_cache.clear(), self.v_cache.clear()
        for i, L in enumerate(self.cfg.layer_specs):
            gk, dk, gv, dv = _pool_heads(L.mixer)
            self.k_cache[i] = torch.zeros(num_blocks, gk, self.bs, dk, dtype=self.dtype, device=self.dev)
            self.v_cache[i] = torch.zeros(num_blocks, gv, self.bs, dv, dtype=self.dtype, device=self.dev)

    def alloc_state(self, max_num_seqs: int) -> None:
        """Per live sequence the token before its next one, and one fp32 matrix state [H, dk, dv] per parallel layer.  Slots are
        never cleared: a sequence that starts at position 0 ignores their contents."""
        self.max_num_seqs = int(max_num_seqs)
        self.state.clear()
        self.last_token = torch.zeros(max_num_seqs, dtype=torch.int64, device=self.dev)
        for i, L in enumerate(self.cfg.layer_specs):
            if isinstance(L.mixer, ParallelSpec):
                r = L.mixer.right
                self.state[i] = torch.zeros(max_num_seqs, r.heads, r.dim, r.vdim, dtype=torch.float32, device=self.dev)

    def prepare_decode(self, max_batch: int, max_nb: int) -> None:
        """Static index tensors of the decode-only batch (one row per sequence)."""
        if self._arange.shape[0] < max_batch + 1:
            self._arange = torch.arange(max_batch + 1, dtype=torch.int32, device=self.dev)

    def decode_schedule(self, seq_lens_host) -> int:
        return 0

    # ------------------------------------------------------------------ forward
    def _window(self, li: int, m: WindowSpec, proj: torch.Tensor, positions, slots, batch: ops.SeqBatch) -> torch.Tensor:
        w, p, kc, vc = self.w, f"l{li}.mix", self.k_cache[li], self.v_cache[li]
        q = ops.qk_rope_cache(proj, m.heads, m.kv_heads, m.dim, m.dim, positions, self.rot[m.rot], m.rot.dims, slots, kc, vc,
                              v_from_k=True, q_norm=w[p + ".q.norm"], k_norm=w[p + ".k.norm"], eps=self.cfg.eps)
        o = ops.chunk_attention(q, kc, vc, batch, m.scale, window=m.window, sink=1.0, sink_logits=w[p + ".sink"], softcap=m.softcap)
        return torch.nn.functional.linear(o.view(proj.shape[0], -1), w[p + ".o"], w[p + ".o.b"])

    def _differential(self, li: int, m: DiffSpec, proj: torch.Tensor, positions, slots, batch: ops.SeqBatch) -> torch.Tensor:
        kc, vc = self.k_cache[li], self.v_cache[li]
        q = ops.qk_rope_cache(proj, 2 * m.heads, 2 * m.kv_heads, m.dim, m.vdim, positions, self.rot[m.rot], m.rot.dims, slots, kc, vc)
        o = ops.chunk_attention(q, kc, vc, batch, m.scale, window=m.window, keep_first=m.keep_first, maps=2, map_lambda=self.lam[li],
                                map_eps=self.cfg.eps, map_scale=1.0 - m.diff)
        return torch.nn.functional.linear(o.view(proj.shape[0], -1), self.w[f"l{li}.mix.o"])

    def _parallel(self, li: int, m: ParallelSpec, proj: torch.Tensor, positions, slots, batch: ops.SeqBatch) -> Tuple[torch.Tensor, torch.Tensor]:
        """The two halves' outputs, before their norms."""
        w, p, cols = self.w, f"l{li}.mix", self.cols[li]
        a, r, T = m.left, m.right, proj.shape[0]

        def right() -> torch.Tensor:                 # retention over the state slots
            qkv, _, decay = ops.recur_prep(proj[:, cols["right"]:], r.heads, r.heads, r.dim, r.vdim, batch, k_scale=r.dim ** -0.5,
                                           decay_mode=ops.DECAY_HEAD_CONST, decay_bias=w[p + ".right.decay"], cos_sin=self.rot[r.rot])
            s = ops.channel_scan(qkv, None, decay, r.heads, r.heads, r.dim, r.vdim, batch, self.state[li], delta=False)
            o = ops.gated_head_norm(s, proj[:, cols["g"]:cols["g"] + r.heads * r.vdim], None, self.cfg.eps, ops.GATE_SILU)
            return torch.nn.functional.linear(o, w[p + ".right.o"])

        main = torch.cuda.current_stream(self.dev)
        if self.overlap:
            self._side.wait_stream(main)             # proj exists; what an earlier layer left of its halves has been read
            with torch.cuda.stream(self._side):
                y2 = right()
        kc, vc = self.k_cache[li], self.v_cache[li]
        q = ops.qk_rope_cache(proj[:, cols["left"]:], a.heads, a.kv_heads, a.dim, a.vdim, positions, self.rot[a.rot], a.rot.dims, slots,
                              kc, vc)
        o = ops.chunk_attention(q, kc, vc, batch, a.scale, a.chunk)
        y1 = torch.nn.functional.linear(o.view(T, -1), w[p + ".left.o"], w[p + ".left.o.b"])
        if self.overlap:
            main.wait_stream(self._side)
        else:
            y2 = right()
        return y1, y2

    def _mlp(self, li: int, f: Union[DenseSpec, ExpertsSpec], h: torch.Tensor) -> torch.Tensor:
        w, p, lin = self.w, f"l{li}.mlp", torch.nn.functional.linear
        if isinstance(f, DenseSpec):
            return lin(ops.glu_and_mul(lin(h, w[p + ".gate_up"]), ops.GLU_CLAMPED, GLU_ALPHA, f.limit), w[p + ".down"])
        shared = None
        if f.shared_ff:
            shared = lin(ops.glu_and_mul(lin(h, w[p + ".shared.gate_up"]), ops.GLU_SILU), w[p + ".shared.down"])
        ids, wts = ops.moe_route(h, w[p + ".router"], None, f.top, scoring=ops.ROUTE_SIGMOID_PLAIN)
        gu = w[p + ".gate_up"]
        return ops.moe_experts(h, ids, wts, gu[:, :f.ff], gu[:, f.ff:], w[p + ".down"], w_gate_up=gu, weight_on_input=True, add=shared)

    def forward(self, tokens: torch.Tensor, positions: torch.Tensor, slots: torch.Tensor, n_decode: int,
                dec_block_tables: Optional[torch.Tensor], dec_seq_lens: Optional[torch.Tensor], prefill,
                sample_rows: Optional[torch.Tensor], num_splits: int = 0,
                dec_state_slots: Optional[torch.Tensor] = None) -> torch.Tensor:
        """tokens int64 [T] (rows [0, n_decode) = one new token per running sequence, the rest = prompt chunks),
        positions int32 [T], slots int64 [T] (cache slot of every row).  Returns logits [len(sample_rows) or T, vocab]
        in the model's dtype."""
        c, w = self.cfg, self.w
        if n_decode and self._arange.shape[0] < n_decode + 1:
            self._arange = torch.arange(n_decode + 1, dtype=torch.int32, device=self.dev)
        if n_decode and dec_state_slots is None:
            raise ValueError("decode rows need their state slots")
        if prefill is not None and prefill.total_tokens and prefill.state_slots is None:
            raise ValueError("prompt chunks need their state slots")
        batch = ops.step_batch(self._arange, n_decode, dec_block_tables, dec_seq_lens, dec_state_slots, prefill)
        T, D, n, rms = tokens.shape[0], c.hidden, len(c.layer_specs), ops.NORM_RMS
        if c.buckets:                                                                # the fp32 residual
            x = ops.embed_bigram(w["embed"], w["bigram"], tokens, batch, c.mul_prev, c.mul_cur, self.last_token)
        else:
            x = ops.embed_streams(w["embed"], tokens, 1, 1.0).view(T, D)
        h = ops.sandwich_norm(x, pre_w=w["l0.norm1"], eps=c.eps, norm_kind=rms, h_dtype=self.dtype)
        for li in range(n):
            L, p = c.layer_specs[li], f"l{li}"
            m, post = L.mixer, w[p + ".norm1b"]
            nxt = w[f"l{li + 1}.norm1"] if li + 1 < n else None     # a sublayer's write-back and the next one's norm in one pass
            pre = w[p + ".norm2"] if L.mlp is not None else nxt
            proj = torch.nn.functional.linear(h, w[p + ".wproj"], w.get(p + ".bproj"))
            if isinstance(m, ParallelSpec):
                y1, y2 = self._parallel(li, m, proj, positions, slots, batch)
                h = ops.sandwich_norm_pair(x, y1, w[p + ".mix.left.out"], y2, w[p + ".mix.right.out"], PAIR_SCALE, post, pre, c.eps)
            else:
                mix = self._window if isinstance(m, WindowSpec) else self._differential
                h = ops.sandwich_norm(x, mix(li, m, proj, positions, slots, batch), post, None, pre, eps=c.eps, norm_kind=rms)
            if L.mlp is not None:
                h = ops.sandwich_norm(x, self._mlp(li, L.mlp, h), w[p + ".norm2b"], None, nxt, eps=c.eps, norm_kind=rms)
            if self.capture is not None:
                self.capture.append(x.clone())
        if sample_rows is not None:
            x = x.index_select(0, sample_rows).contiguous()
        h = ops.sandwich_norm(x, pre_w=w["final.norm"], eps=c.eps, norm_kind=rms, h_dtype=self.dtype)
        return torch.nn.functional.linear(h, w["head"])
