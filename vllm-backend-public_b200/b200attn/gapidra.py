"""Gapidra decoder on the b200attn ops: parallel layers -- one RMS norm per layer whose output both the sequence mixer and the
feed-forward read, x <- x + (mixer(h) + ff(h)) around one fp32 residual -- with one of two mixers per layer:

  latent_attention   sliding-window softmax attention over one low-rank latent per token that all heads share plus one shared
                     rotated key part (pairs (i, i + rot_dim / 2)), a learned sink per head in the denominator, a sigmoid gate
                     per output channel.
  attention          sliding-window grouped-query attention whose weights are sigmoids of the scores plus a bias per head, not
                     normalised over the keys; q and k are RMS-normed over the whole projection, then partly rotated
                     (pairs (2i, 2i + 1), YaRN frequency scaling).

The feed-forward is dense with xIELU (quadratic above zero, exponential below, both curvatures learned), or absent.

The parallel form shapes the work of a layer: everything that reads h (queries, keys / values or their latent, the output
gate, the feed-forward's up rows) is ONE product, and W_o and W_down are ONE product over the concatenated columns
[gated heads | activated units], so that the sum of the two sublayers is formed in its fp32 accumulator.

The model plugs into the same engine as the other families (b200attn.engine.LLMEngine): paged pools addressed through the
scheduler's block tables and slot mapping, one forward over [decode rows | prompt chunks], logits for the sampled rows.
Projections and the vocabulary head are library GEMMs (torch -> cuBLAS); everything between them is this repo's kernels
(csrc/post_norm.cu, chunk_attention.cu, latent_attention.cu).  There is no CPU path.

Every size, the layer order and every constant come from the checkpoint's config.json (`architecture: "Gapidra"`);
weights from its *.safetensors, or random from a seed.
"""
from __future__ import annotations

import json
import math
from dataclasses import dataclass
from pathlib import Path
from typing import Dict, List, Optional, Tuple, Union

import torch

from . import ops

ARCHITECTURE = "Gapidra"
# A step with at least this many prompt rows rebuilds keys and values per head for them in its latent layers (bf16):
# (dim + rot_dim + vdim) multiplications per (query, key, head) instead of (2 kv_rank + rot_dim) in the latent space, for
# two more GEMMs per layer over the rows the portions can see.  Decode rows and short portions stay in the latent space.
PROMPT_PER_HEAD_MIN_ROWS = 256
PROMPT_PER_HEAD_MAX_CONTEXT = 4      # ... unless the visible rows outnumber the prompt rows by more than this factor


@dataclass(frozen=True)
class Rotation:
    dims: int = 0              # how many leading entries turn (the rest pass)
    base: float = 10000.0
    scaling: Optional[Tuple[Tuple[str, float], ...]] = None     # sorted items of {factor, original, fast, slow}


@dataclass(frozen=True)
class LatentSpec:
    heads: int
    dim: int                   # per-head unrotated query / key size
    rot_dim: int               # per-head rotated query size = size of the shared rotated key part
    vdim: int
    kv_rank: int               # latent size
    scale: float
    window: int                # a query sees its own position and the window - 1 before it (0: plain causal)
    rot: Rotation

    @property
    def row(self) -> int:
        return self.kv_rank + self.rot_dim

    @property
    def out(self) -> int:
        return self.heads * self.vdim


@dataclass(frozen=True)
class SigmoidSpec:
    heads: int
    kv_heads: int
    dim: int
    vdim: int
    scale: float
    window: int
    rot: Rotation

    @property
    def out(self) -> int:
        return self.heads * self.vdim


@dataclass(frozen=True)
class DenseSpec:
    ff: int


MixerSpec = Union[LatentSpec, SigmoidSpec]


@dataclass(frozen=True)
class LayerSpec:
    mixer: MixerSpec
    mlp: Optional[DenseSpec]


def layer_tensors(p: str, L: LayerSpec, D: int) -> Dict[str, Tuple[int, ...]]:
    """Name -> shape of one layer's tensors."""
    m, q = L.mixer, p + ".mix"
    out: Dict[str, Tuple[int, ...]] = {p + ".norm1": (D,)}
    if isinstance(m, LatentSpec):
        out.update({q + ".q": (m.heads * (m.dim + m.rot_dim), D), q + ".dkv": (m.row, D), q + ".dkv.norm": (m.kv_rank,),
                    q + ".uk": (m.heads * m.dim, m.kv_rank), q + ".uv": (m.out, m.kv_rank), q + ".sink": (m.heads,),
                    q + ".g": (m.out, D)})
    else:
        nq, nk = m.heads * m.dim, m.kv_heads * m.dim
        out.update({q + ".q": (nq, D), q + ".k": (nk, D), q + ".v": (m.kv_heads * m.vdim, D), q + ".q.norm": (nq,),
                    q + ".k.norm": (nk,), q + ".pb": (m.heads,)})
    out[q + ".o"] = (D, m.out)
    if L.mlp is not None:
        out.update({p + ".mlp.up": (L.mlp.ff, D), p + ".mlp.down": (D, L.mlp.ff), p + ".mlp.act": (2,)})
    return out


@dataclass
class GapidraConfig:
    name: str
    vocab: int
    hidden: int
    layer_specs: List[LayerSpec]
    eps: float = 1e-6
    embed_scale: float = 1.0
    max_position: int = 1 << 20            # the rotary tables are built for the engine's max_model_len
    family: str = "gapidra"

    @property
    def layers(self) -> int:
        return len(self.layer_specs)

    def tensors(self) -> Dict[str, Tuple[int, ...]]:
        """Name -> shape of every tensor of a checkpoint of this configuration."""
        D = self.hidden
        out: Dict[str, Tuple[int, ...]] = {"embed": (self.vocab, D), "final.norm": (D,), "head": (self.vocab, D)}
        for i, L in enumerate(self.layer_specs):
            out.update(layer_tensors(f"l{i}", L, D))
        return out

    @property
    def params(self) -> int:
        return sum(math.prod(s) for s in self.tensors().values())

    def kv_bytes_per_token(self, kv_elem_bytes: int = 2, tp: int = 1) -> int:
        return sum((m.row if isinstance(m, LatentSpec) else m.kv_heads * (m.dim + m.vdim)) * kv_elem_bytes
                   for m in (L.mixer for L in self.layer_specs))

    def state_bytes_per_seq(self, elem_bytes: int = 2) -> int:
        return 0                                     # attention only: nothing is kept per sequence besides the pools

    def activation_bytes(self, tokens: int, seqs: int, elem_bytes: int = 2) -> int:
        wide = [self.hidden]
        for L in self.layer_specs:
            m, ff = L.mixer, L.mlp.ff if L.mlp is not None else 0
            if isinstance(m, LatentSpec):
                # projection row, absorbed queries and latent outputs; gathered rows with their per-head keys and values
                wide.append(m.heads * (2 * m.dim + 2 * m.rot_dim + 2 * m.kv_rank + 3 * m.vdim) + m.row + 2 * ff
                            + PROMPT_PER_HEAD_MAX_CONTEXT * (m.row + m.heads * (m.dim + m.vdim)))
            else:
                wide.append((2 * m.heads + m.kv_heads) * m.dim + (m.heads + m.kv_heads) * m.vdim + 2 * ff)
        return tokens * (self.hidden * 8 + 2 * max(wide) * elem_bytes) + seqs * self.vocab * 8 + (1 << 28)

    def build_model(self, device, **kw):
        return GapidraModel(self, device, **kw)


def _rotation(m: dict, width: int, where: str) -> Rotation:
    rot = m.get("rot")
    if not rot:
        return Rotation()
    s = rot.get("scaling")
    r = Rotation(int(rot.get("dims", width)), float(rot.get("base", 10000.0)),
                 tuple(sorted((k, float(v)) for k, v in s.items())) if s else None)
    if r.dims % 2 or not 0 <= r.dims <= width:
        raise ValueError(f"{where}: rot.dims {r.dims} must be even and at most {width}")
    if r.scaling and not {"factor", "original", "fast", "slow"} <= {k for k, _ in r.scaling}:
        raise ValueError(f"{where}: rot.scaling needs factor, original, fast and slow")
    return r


def config_from_dict(c: dict, name: str = ARCHITECTURE) -> GapidraConfig:
    """config.json -> GapidraConfig.  Keys: vocab, width, norm.eps, embedding.scale, layers [{type, mixer, mlp null | {kind:
    dense, ff}}] with the mixers
      latent_attention  {heads, dim, rot_dim, vdim, kv_rank, scale, mask {size}, rot {base, dims (= rot_dim), scaling}}
      attention         {heads, kv_heads, dim, vdim, scale, mask {size}, rot {base, dims, scaling {factor, original, fast, slow}}}."""
    specs: List[LayerSpec] = []
    for i, L in enumerate(c["layers"]):
        where, kind, m = f"layer {i}", L["type"], L["mixer"]
        window = int((m.get("mask") or {}).get("size") or 0)
        if window < 0:
            raise ValueError(f"{where}: mask.size {window} is negative")
        if kind == "latent_attention":
            rot_dim = int(m["rot_dim"])
            mixer: MixerSpec = LatentSpec(int(m["heads"]), int(m["dim"]), rot_dim, int(m["vdim"]), int(m["kv_rank"]),
                                          float(m["scale"]), window, _rotation(m, rot_dim, where))
        elif kind == "attention":
            dim = int(m["dim"])
            mixer = SigmoidSpec(int(m["heads"]), int(m.get("kv_heads", m["heads"])), dim, int(m.get("vdim", dim)),
                                float(m["scale"]), window, _rotation(m, dim, where))
            if mixer.kv_heads < 1 or mixer.heads % mixer.kv_heads:
                raise ValueError(f"{where}: {mixer.heads} query heads over {mixer.kv_heads} key/value heads")
        else:
            raise ValueError(f"{where}: unknown mixer type {kind!r}")
        f = L.get("mlp")
        if f and f.get("kind") != "dense":
            raise ValueError(f"{where}: unknown feed-forward kind {f.get('kind')!r}")
        specs.append(LayerSpec(mixer, DenseSpec(int(f["ff"])) if f else None))
    return GapidraConfig(name=name, vocab=int(c["vocab"]), hidden=int(c["width"]), layer_specs=specs,
                         eps=float((c.get("norm") or {}).get("eps", 1e-6)),
                         embed_scale=float((c.get("embedding") or {}).get("scale", 1.0)))


def config_from_dir(path: Path) -> GapidraConfig:
    path = Path(path)
    return config_from_dict(json.loads((path / "config.json").read_text()), name=path.name)


def bench_config(hidden: int, layers: int, heads: int, kv_heads: int, head_dim: int, ff: int, vocab: int, kv_rank: int = 512,
                 rot_dim: int = 64, window: int = 1024, name: str = "gapidra-bench") -> GapidraConfig:
    """A model-sized geometry for benchmarks: latent and sigmoid layers in turn, every layer with a feed-forward."""
    yarn = (("factor", 8.0), ("fast", 32.0), ("original", 4096.0), ("slow", 1.0))
    specs = []
    for i in range(layers):
        m: MixerSpec
        if i % 2 == 0:
            m = LatentSpec(heads, head_dim, rot_dim, head_dim, kv_rank, (head_dim + rot_dim) ** -0.5, window, Rotation(rot_dim, 1e4))
        else:
            m = SigmoidSpec(heads, kv_heads, head_dim, head_dim, head_dim ** -0.5, window, Rotation(head_dim // 2, 1e6, yarn))
        specs.append(LayerSpec(m, DenseSpec(ff)))
    return GapidraConfig(name, vocab, hidden, specs, embed_scale=hidden ** 0.5)


class GapidraModel:
    """Weights + per-layer pools + forward over one scheduled token batch.  One instance per GPU."""

    supports_fp32 = True
    launches_per_layer = 6

    def __init__(self, cfg: GapidraConfig, device: torch.device, num_blocks: int, block_size: int = 16, seed: int = 0,
                 weights_dir: Optional[Path] = None, max_position: Optional[int] = None,
                 kv_dtype: torch.dtype = torch.bfloat16, tp=None, dtype: torch.dtype = torch.bfloat16,
                 max_num_seqs: int = 1):
        if device.type != "cuda":
            raise ValueError("GapidraModel needs a CUDA device (b200attn has no CPU path)")
        if tp is not None and tp.size > 1:
            raise ValueError("Gapidra runs on one GPU per replica: tensor_parallel_size must be 1")
        if dtype not in (torch.bfloat16, torch.float32):
            raise ValueError(f"dtype {dtype}: bfloat16 or float32")
        if kv_dtype not in (torch.bfloat16, dtype):
            raise ValueError("Gapidra keeps its pools in the activation type (no fp8 cache)")
        self.cfg, self.dev, self.bs, self.dtype = cfg, device, block_size, dtype
        self.tp, self.tp_size, self.tp_rank = None, 1, 0
        self.vocab_parallel = False
        self.Hq = self.Hkv = 0                      # no paged-decode schedule to plan
        self.max_position = max_position or min(cfg.max_position, 1 << 17)
        self.max_num_seqs = max_num_seqs
        self.w: Dict[str, torch.Tensor] = {}
        self.cols: List[Dict[str, int]] = []        # per layer: first column of every part of its fused projection
        self.xielu: List[Tuple[float, float]] = []  # per layer: the curvatures above and below zero
        if weights_dir is not None and any(Path(weights_dir).glob("*.safetensors")):
            self._load(Path(weights_dir))
        else:
            self._random_init(seed)
        self._fuse()
        # one rotary table per distinct (dims, base, scaling); both pair layouts read the same table
        self.rot: Dict[Rotation, torch.Tensor] = {}
        for L in cfg.layer_specs:
            r = L.mixer.rot
            if r not in self.rot:
                self.rot[r] = ops.rotary_table(self.max_position, r.dims, r.base, dict(r.scaling) if r.scaling else None, device) \
                    if r.dims else torch.zeros(self.max_position, 0, dtype=torch.float32, device=device)
        self.num_blocks = 0
        self.k_cache: Dict[int, torch.Tensor] = {}
        self.v_cache: Dict[int, torch.Tensor] = {}
        self.latent_cache: Dict[int, torch.Tensor] = {}
        self.alloc_cache(num_blocks)
        self._arange = torch.arange(max_num_seqs + 1, dtype=torch.int32, device=device)
        self.capture: Optional[list] = None         # tests: set to a list to collect the residual after every layer

    # ------------------------------------------------------------------ weights
    def _random_init(self, seed: int) -> None:
        g = torch.Generator(device=self.dev).manual_seed(seed)
        raw = {}
        for name, shape in self.cfg.tensors().items():
            t = torch.randn(*shape, generator=g, device=self.dev, dtype=torch.float32)
            if name.endswith(".pb"):
                t = t - 3.0
            elif name.endswith(".act"):
                t = 0.5 * t
            elif len(shape) == 1 and not name.endswith(".sink"):
                t = 1.0 + 0.1 * t
            elif len(shape) == 2 and name != "embed":
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
        """Matrices in the activation type, parameter vectors in fp32."""
        for k, t in raw.items():
            self.w[k] = t.to(torch.float32 if t.dim() == 1 else self.dtype).contiguous()

    def _stack(self, parts: List[Tuple[str, List[torch.Tensor]]]) -> Tuple[torch.Tensor, Dict[str, int]]:
        """Rows of several matrices as one projection matrix; every named part starts on a multiple of eight rows (zero rows
        between), so that the columns it produces stay 16-byte aligned.  Returns the matrix and the parts' first columns."""
        rows, cols, at = [], {}, 0
        for name, mats in parts:
            cols[name] = at
            n = sum(m.shape[0] for m in mats)
            rows += mats
            if n % 8:
                rows.append(torch.zeros(-n % 8, mats[0].shape[1], dtype=self.dtype, device=self.dev))
            at += n + -n % 8
        return torch.cat(rows).contiguous(), cols

    def _fuse(self) -> None:
        """Per layer: ONE matrix for everything that reads the norm's output (latent: q | gate | down-projection; attention:
        q k v; then the feed-forward's up rows) and ONE for what is added to the residual ([W_o | W_down] side by side), the
        latent's up-projections per head, the two curvatures of xIELU."""
        w, c = self.w, self.cfg
        for i, L in enumerate(c.layer_specs):
            p, m, q = f"l{i}", L.mixer, f"l{i}.mix"
            if isinstance(m, LatentSpec):
                parts = [("q", [w.pop(q + ".q")]), ("g", [w.pop(q + ".g")]), ("dkv", [w.pop(q + ".dkv")])]
                w[q + ".uk"] = w[q + ".uk"].view(m.heads, m.dim, m.kv_rank)                                      # q_h -> latent space
                w[q + ".uv"] = w[q + ".uv"].view(m.heads, m.vdim, m.kv_rank).transpose(1, 2).contiguous()        # [H, R, dv]
            else:
                parts = [("qkv", [w.pop(q + ".q"), w.pop(q + ".k"), w.pop(q + ".v")])]
            out = [w.pop(q + ".o")]
            curv = (0.0, 0.0)
            if L.mlp is not None:
                parts.append(("up", [w.pop(p + ".mlp.up")]))
                out.append(w.pop(p + ".mlp.down"))
                above, below = torch.nn.functional.softplus(w.pop(p + ".mlp.act").double()).tolist()
                curv = (above, 0.5 + below)
            w[p + ".wproj"], cols = self._stack(parts)
            w[p + ".wout"] = torch.cat(out, dim=1).contiguous()
            self.cols.append(cols)
            self.xielu.append(curv)

    def weight_bytes(self) -> int:
        return sum(t.numel() * t.element_size() for t in self.w.values())

    # ------------------------------------------------------------------ caches
    def alloc_cache(self, num_blocks: int) -> None:
        """Per latent layer one pool [num_blocks, bs, kv_rank + rot_dim]; per attention layer a K pool (normed, rotated keys)
        [num_blocks, G, bs, dk] and a V pool [num_blocks, G, bs, dv]."""
        self.num_blocks = int(num_blocks)
        self.k_cache.clear(), self.v_cache.clear(), self.latent_cache.clear()
        for i, L in enumerate(self.cfg.layer_specs):
            m = L.mixer
            if isinstance(m, LatentSpec):
                self.latent_cache[i] = torch.zeros(num_blocks, self.bs, m.row, dtype=self.dtype, device=self.dev)
            else:
                self.k_cache[i] = torch.zeros(num_blocks, m.kv_heads, self.bs, m.dim, dtype=self.dtype, device=self.dev)
                self.v_cache[i] = torch.zeros(num_blocks, m.kv_heads, self.bs, m.vdim, dtype=self.dtype, device=self.dev)

    def alloc_state(self, max_num_seqs: int) -> None:
        """Nothing is kept per sequence besides the pools."""
        self.max_num_seqs = int(max_num_seqs)

    def prepare_decode(self, max_batch: int, max_nb: int) -> None:
        """Static index tensors of the decode-only batch (one row per sequence)."""
        if self._arange.shape[0] < max_batch + 1:
            self._arange = torch.arange(max_batch + 1, dtype=torch.int32, device=self.dev)

    def decode_schedule(self, seq_lens_host) -> int:
        return 0

    # ------------------------------------------------------------------ forward
    def _prompt_plans(self, prefill) -> Dict[int, tuple]:
        """Window -> (rows N, cu_k, k_lo) of the pool rows the step's prompt portions see in a latent layer of that window.
        Layers whose window is not listed keep every row in the latent space."""
        if prefill is None or self.dtype != torch.bfloat16 or prefill.total_tokens < PROMPT_PER_HEAD_MIN_ROWS \
                or prefill.q_lens_host is None or prefill.kv_lens_host is None:
            return {}
        plans = {}
        for L in self.cfg.layer_specs:
            m = L.mixer
            if isinstance(m, LatentSpec) and m.window not in plans:
                one = ops.latent_prompt_plan(prefill.q_lens_host, prefill.kv_lens_host, m.window,
                                             PROMPT_PER_HEAD_MAX_CONTEXT * prefill.total_tokens, self.dev)
                if one is not None:
                    plans[m.window] = one
        return plans

    def _latent(self, li: int, m: LatentSpec, proj: torch.Tensor, joint: torch.Tensor, positions: torch.Tensor,
                slots: torch.Tensor, batch: ops.SeqBatch, n_decode: int, prefill, plans: Dict[int, tuple]):
        """Writes the gated heads of the rows on the per-head path into joint; returns the heads [n, H * dv] and gates of the
        first n rows, which stayed in the latent space and are still to be gated (None: no such rows)."""
        w, p, cols = self.w, f"l{li}.mix", self.cols[li]
        H, dn, dr, dv, R = m.heads, m.dim, m.rot_dim, m.vdim, m.kv_rank
        T = proj.shape[0]
        cache, sink = self.latent_cache[li], w[p + ".sink"]
        qa = ops.latent_prep(proj, H, dn, dr, m.rot.dims, R, cols["q"], cols["dkv"], w[p + ".dkv.norm"], self.cfg.eps, positions,
                             self.rot[m.rot], slots, cache, interleaved=False)
        qh = proj[:, cols["q"]:cols["q"] + H * (dn + dr)].view(T, H, dn + dr)
        gate = proj[:, cols["g"]:cols["g"] + m.out]
        plan = plans.get(m.window)
        if plan is not None and not (ops.window_attention_ok(self.dtype, dn, dr, dv) and m.row % 8 == 0 and joint.stride(0) % 8 == 0):
            plan = None
        nl = T if plan is None else n_decode            # rows that stay in the latent space
        if plan is not None:
            # long prompt portions: keys and values per head, rebuilt over the pool rows the portions see
            N, cu_k, k_lo = plan
            npf = len(prefill.q_lens_host)
            lat = ops.latent_gather(cache, prefill.block_tables, cu_k, k_lo, npf, N)
            kn = torch.nn.functional.linear(lat[:, :R], w[p + ".uk"].view(H * dn, R)).view(N, H, dn)
            v = torch.empty(N, H, dv, dtype=proj.dtype, device=proj.device)
            torch.bmm(lat[:, :R].unsqueeze(0).expand(H, N, R), w[p + ".uv"], out=v.transpose(0, 1))
            ops.window_attention(qh[nl:, :, :dn], qa[nl:, :, R:], kn, lat[:, R:], v, prefill.cu_q, prefill.ctx_start, cu_k, k_lo,
                                 npf, m.scale, m.window, gate=gate[nl:], sink_logits=sink, out=joint[nl:, :m.out])
        if not nl:
            return None, None
        # the unrotated part of every query head, carried into the latent space: qa[:, h, :R] = q_h W_uk[h]
        torch.bmm(qh[:nl, :, :dn].transpose(0, 1), w[p + ".uk"], out=qa[:nl, :, :R].transpose(0, 1))
        lb = batch if plan is None else ops.SeqBatch(batch.cu_q[:nl + 1], batch.ctx_start[:nl], batch.block_tables[:nl], None, nl, nl)
        o = ops.latent_attention(qa[:nl], cache, lb, R, m.scale, m.window, sink_logits=sink)
        ov = torch.empty(nl, H, dv, dtype=proj.dtype, device=proj.device)
        torch.bmm(o.transpose(0, 1), w[p + ".uv"], out=ov.transpose(0, 1))       # head outputs = W_uv[h] (sum_j p_j c_j)
        return ov.view(nl, m.out), gate[:nl]

    def _sigmoid(self, li: int, m: SigmoidSpec, proj: torch.Tensor, joint: torch.Tensor, positions: torch.Tensor,
                 slots: torch.Tensor, batch: ops.SeqBatch) -> None:
        """Writes the heads into joint's first columns."""
        w, p = self.w, f"l{li}.mix"
        k_cache, v_cache = self.k_cache[li], self.v_cache[li]
        q = ops.qk_rope_cache(proj, m.heads, m.kv_heads, m.dim, m.vdim, positions, self.rot[m.rot], m.rot.dims, slots, k_cache,
                              v_cache, interleaved=True, q_norm=w[p + ".q.norm"], k_norm=w[p + ".k.norm"], eps=self.cfg.eps)
        ops.chunk_attention(q, k_cache, v_cache, batch, m.scale, window=m.window, weight_kind=ops.WEIGHT_SIGMOID,
                            head_bias=w[p + ".pb"], out=joint[:, :m.out])

    def _layer(self, li: int, h: torch.Tensor, positions, slots, batch, n_decode, prefill, plans) -> torch.Tensor:
        """mixer(h) + ff(h)."""
        L, w, p, cols = self.cfg.layer_specs[li], self.w, f"l{li}", self.cols[li]
        m, ff = L.mixer, L.mlp.ff if L.mlp is not None else 0
        proj = torch.nn.functional.linear(h, w[p + ".wproj"])
        joint = torch.empty(h.shape[0], m.out + ff, dtype=h.dtype, device=h.device)
        heads = gate = None
        if isinstance(m, LatentSpec):
            heads, gate = self._latent(li, m, proj, joint, positions, slots, batch, n_decode, prefill, plans)
        else:
            self._sigmoid(li, m, proj, joint, positions, slots, batch)
        if ff or heads is not None:
            up = proj[:, cols["up"]:cols["up"] + ff] if ff else None
            ops.parallel_join(joint, heads, gate, m.out, up, ops.FF_XIELU, *self.xielu[li])
        return torch.nn.functional.linear(joint, w[p + ".wout"])

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
        batch = ops.step_batch(self._arange, n_decode, dec_block_tables, dec_seq_lens, None, prefill)
        plans = self._prompt_plans(prefill)
        T, D, n = tokens.shape[0], c.hidden, len(c.layer_specs)
        x = ops.embed_streams(w["embed"], tokens, 1, c.embed_scale).view(T, D)       # the fp32 residual
        h = ops.sandwich_norm(x, pre_w=w["l0.norm1"], eps=c.eps, norm_kind=ops.NORM_RMS, h_dtype=self.dtype)
        for li in range(n):
            y = self._layer(li, h, positions, slots, batch, n_decode, prefill, plans)
            nxt = w[f"l{li + 1}.norm1"] if li + 1 < n else None       # residual add and the next layer's norm in one pass
            h = ops.sandwich_norm(x, y, pre_w=nxt, eps=c.eps, norm_kind=ops.NORM_RMS)
            if self.capture is not None:
                self.capture.append(x.clone())
        if sample_rows is not None:
            x = x.index_select(0, sample_rows).contiguous()
        h = ops.sandwich_norm(x, pre_w=w["final.norm"], eps=c.eps, norm_kind=ops.NORM_RMS, h_dtype=self.dtype)
        return torch.nn.functional.linear(h, w["head"])
