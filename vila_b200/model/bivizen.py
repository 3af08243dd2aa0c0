"""Bivizen: a decoder-only language model of recurrent and attention mixers with parallel sublayers on the
ragged-batch kernels.

Residual stream x (fp32).  Layer i:  h = rms(x) * norm1,  x += ls1 * mixer(h) + ls2 * ff(h)  (both sublayers read the one
normed h; ls1 / ls2 are per-channel scales; a layer may have no feed-forward), rms(v) = v / sqrt(mean(v^2) + eps).
Mixers (config `layers[i].type`):

  attention   grouped-query heads with biased q / k / v projections; rotary positions on the first `rot.dims` columns of
              q and k in the halves layout; scores times `scale`, bounded to softcap * tanh(s / softcap); causal softmax;
              a layer with `v_mix` caches (1 - l) v + l v_first, where v_first are the first such layer's values of the
              same token and l is the layer's number; per-head sigmoid output gate
  delta       gated delta rule: causal convolution (`conv` taps) + SiLU on q, k, v, unit q and k, a decay and a step size
              per head, state [dim, vdim] per head, per-head RMS norm of the read-out times silu of a gate projection
  gla         gated linear attention: a decay per key channel sigmoid(z)^(1 / tau) from a low-rank projection, state and
              read-out as above, no convolution

Feed-forward: a clamped gated unit  min(g, L) * sigmoid(1.702 min(g, L)) * (clamp(u, -L, L) + 1).

One step takes a RaggedBatch and a HybridCache owned by the serving engine (vila_b200/serving.py): attention layers keep
k | v rows in a paged pool, recurrent ones their state (and the convolution's last inputs) in the sequence's slot.
dtype bfloat16: projections on the tcgen05 GEMM (shapes it does not take go to the CUDA-core grouped kernel), convolution
outputs in bf16; positions and angles, norms, scores and softmax, decays, step sizes, unit norms, states and the residual
sum in fp32.  dtype float32: the same kernels with fp32 tensors and the CUDA-core linear layer throughout.
"""
from __future__ import annotations

import json
from dataclasses import dataclass, field
from pathlib import Path
from typing import Dict, List, Optional, Tuple

import torch

from .. import ops
from .ludazen import RotaryConfig
from .moronex import read_safetensors, stack_rows

ARCHITECTURE = "Bivizen"
GLU_ALPHA = 1.702    # fixed by the architecture: slope of the sigmoid inside the gated unit
UNIT_EPS = 1e-6      # fixed by the architecture: added to the sum of squares of q and k of the delta rule


@dataclass
class BivizenLayerConfig:
    type: str                         # "attention" | "delta" | "gla"
    heads: int
    dim: int
    vdim: int
    kv_heads: int = 0                 # attention: key / value heads; delta: query / key heads
    scale: float = 1.0                # attention
    softcap: float = 0.0              # attention; 0: scores are not capped
    v_mix: bool = False               # attention
    rot: Optional[RotaryConfig] = None
    conv: int = 1                     # delta: taps of the short convolutions
    tau: float = 1.0                  # gla
    ff: int = 0                       # 0: no feed-forward
    limit: float = 0.0


@dataclass
class BivizenConfig:
    vocab: int
    width: int
    norm_eps: float
    layers: List[BivizenLayerConfig] = field(default_factory=list)
    architecture: str = ARCHITECTURE

    @staticmethod
    def from_dict(d: dict) -> "BivizenConfig":
        layers = []
        for i, spec in enumerate(d["layers"]):
            m, kind = spec["mixer"], spec["type"]
            lc = BivizenLayerConfig(type=kind, heads=int(m["heads"]), dim=int(m["dim"]), vdim=int(m["vdim"]))
            if kind == "attention":
                lc.kv_heads, lc.scale = int(m["kv_heads"]), float(m["scale"])
                lc.softcap, lc.v_mix = float(m.get("softcap") or 0.0), bool(m.get("v_mix", False))
                lc.rot = RotaryConfig.from_dict(m["rot"]) if m.get("rot") else RotaryConfig(dims=0, base=1.0)
            elif kind == "delta":
                lc.kv_heads, lc.conv = int(m["kv_heads"]), int(m["conv"])
            elif kind == "gla":
                lc.tau = float(m["tau"])
            else:
                raise ValueError(f"layer {i}: unknown mixer type {kind!r}")
            mlp = spec.get("mlp")
            if mlp is not None:
                if mlp["kind"] != "dense":
                    raise ValueError(f"layer {i}: unknown feed-forward kind {mlp['kind']!r}")
                lc.ff, lc.limit = int(mlp["ff"]), float(mlp["limit"])
            layers.append(lc)
        cfg = BivizenConfig(vocab=int(d["vocab"]), width=int(d["width"]), norm_eps=float(d["norm"]["eps"]), layers=layers)
        cfg.validate()
        return cfg

    def validate(self) -> None:
        mixed = None
        for i, lc in enumerate(self.layers):
            if lc.heads < 1 or lc.dim < 1 or lc.vdim < 1:
                raise ValueError(f"layer {i}: heads {lc.heads}, dim {lc.dim}, vdim {lc.vdim}")
            if lc.type in ("attention", "delta") and (lc.kv_heads < 1 or lc.heads % lc.kv_heads):
                raise ValueError(f"layer {i}: heads {lc.heads} / kv_heads {lc.kv_heads}")
            if lc.type == "attention":
                if lc.rot.dims % 2 or lc.rot.dims > lc.dim or lc.softcap < 0:
                    raise ValueError(f"layer {i}: rot.dims {lc.rot.dims} of {lc.dim}, softcap {lc.softcap}")
                if lc.v_mix:
                    mixed = mixed or (lc.kv_heads, lc.vdim)
                    if (lc.kv_heads, lc.vdim) != mixed:
                        raise ValueError(f"layer {i}: its values {lc.kv_heads} x {lc.vdim} cannot be mixed with the first "
                                         f"mixing layer's {mixed[0]} x {mixed[1]}")
            elif lc.dim > 512:
                raise ValueError(f"layer {i}: a recurrent state of dim {lc.dim} (at most 512)")
            if lc.type == "delta" and not 1 <= lc.conv <= 16:
                raise ValueError(f"layer {i}: conv {lc.conv} not in 1..16")
            if lc.type == "gla" and not lc.tau > 0:
                raise ValueError(f"layer {i}: tau {lc.tau}")

    def to_dict(self) -> dict:
        out = []
        for lc in self.layers:
            m = {"dim": lc.dim, "heads": lc.heads, "vdim": lc.vdim}
            if lc.type == "attention":
                m.update(kv_heads=lc.kv_heads, rot=lc.rot.to_dict(), scale=lc.scale, softcap=lc.softcap, v_mix=lc.v_mix)
            elif lc.type == "delta":
                m.update(conv=lc.conv, kv_heads=lc.kv_heads)
            else:
                m.update(tau=lc.tau)
            out.append({"mixer": m, "mlp": {"ff": lc.ff, "kind": "dense", "limit": lc.limit} if lc.ff else None,
                        "type": lc.type})
        return {"architecture": self.architecture, "layers": out, "norm": {"eps": self.norm_eps}, "vocab": self.vocab,
                "width": self.width}

    def tensor_shapes(self) -> Dict[str, tuple]:
        """name -> shape of every checkpoint tensor (the layout `load_weights` expects); the rank of a decay
        projection is only in the checkpoint and reported as -1 (any)."""
        W, s = self.width, {}
        s["embed"] = (self.vocab, W)
        for i, lc in enumerate(self.layers):
            p, q = f"l{i}.", f"l{i}.mix."
            s[p + "norm1"], s[p + "ls1"] = (W,), (W,)
            if lc.type == "attention":
                for n, rows in (("q", lc.heads * lc.dim), ("k", lc.kv_heads * lc.dim), ("v", lc.kv_heads * lc.vdim)):
                    s[q + n], s[q + n + ".b"] = (rows, W), (rows,)
                if lc.v_mix:
                    s[q + "vmix"] = ()
                s[q + "g"] = (lc.heads, W)
            elif lc.type == "delta":
                for n, rows in (("q", lc.kv_heads * lc.dim), ("k", lc.kv_heads * lc.dim), ("v", lc.heads * lc.vdim)):
                    s[q + n], s[q + n + ".conv"] = (rows, W), (rows, lc.conv)
                s[q + "b"], s[q + "a"] = (lc.heads, W), (lc.heads, W)
                s[q + "A_log"], s[q + "dt_bias"] = (lc.heads,), (lc.heads,)
                s[q + "norm"], s[q + "g"] = (lc.vdim,), (lc.heads * lc.vdim, W)
            else:
                hd = lc.heads * lc.dim
                s[q + "q"], s[q + "k"], s[q + "v"] = (hd, W), (hd, W), (lc.heads * lc.vdim, W)
                s[q + "a1"], s[q + "a2"], s[q + "a2.b"] = (-1, W), (hd, -1), (hd,)
                s[q + "norm"], s[q + "g"] = (lc.vdim,), (lc.heads * lc.vdim, W)
            s[q + "o"] = (W, lc.heads * lc.vdim)
            if lc.ff:
                s[p + "mlp.gate"], s[p + "mlp.up"], s[p + "mlp.down"] = (lc.ff, W), (lc.ff, W), (W, lc.ff)
                s[p + "ls2"] = (W,)
        s["final.norm"], s["head"] = (W,), (self.vocab, W)
        return s


class _Layer:
    """Device tensors of one layer in the layout the kernels want."""


class BivizenForCausalLM:
    """Weights + the per-step compute of the architecture.  Sequences, pages, state slots, batching and
    sampling belong to `vila_b200.serving.TokenEngine`, which calls `forward_step` / `logits`."""

    def __init__(self, cfg: BivizenConfig, device="cuda", dtype=torch.bfloat16):
        assert dtype in (torch.bfloat16, torch.float32)
        cfg.validate()
        self.config, self.device, self.dtype = cfg, torch.device(device), dtype
        self.vocab_size = cfg.vocab
        self.weights: Dict[str, torch.Tensor] = {}
        self.layers: List[_Layer] = []

    # ---- weights ----------------------------------------------------------------------------------
    @classmethod
    def from_pretrained(cls, model_dir, device="cuda", dtype=torch.bfloat16) -> "BivizenForCausalLM":
        d = Path(model_dir)
        cfg = BivizenConfig.from_dict(json.loads((d / "config.json").read_text()))
        files = sorted(d.glob("*.safetensors"))
        if not files:
            raise FileNotFoundError(f"no *.safetensors under {d}")
        tensors: Dict[str, torch.Tensor] = {}
        for f in files:
            tensors.update(read_safetensors(f))
        return cls(cfg, device, dtype).load_weights(tensors)

    def init_random(self, seed: int = 0, scale: float = 1.0, on_device: bool = False, decay_rank: int = 16
                    ) -> "BivizenForCausalLM":
        """Random bf16-representable weights.  on_device: draw them on the model's device (large models)."""
        dev = self.device if on_device else torch.device("cpu")
        g = torch.Generator(device=dev).manual_seed(seed)
        t = {}
        for name, shape in self.config.tensor_shapes().items():
            shape = tuple(decay_rank if n < 0 else n for n in shape)
            last = name.rsplit(".", 1)[-1]
            if last == "vmix":
                v = 0.3 + 0.4 * torch.rand(shape, generator=g, device=dev)
            elif last == "A_log":      # decay rates 1 .. 8
                v = torch.log(1.0 + 7.0 * torch.rand(shape, generator=g, device=dev))
            elif last == "dt_bias":    # step sizes around 0.01 .. 0.1 after softplus
                v = -4.6 + 2.3 * torch.rand(shape, generator=g, device=dev)
            elif last == "conv":
                v = torch.randn(shape, generator=g, device=dev) * 0.5
            elif last in ("ls1", "ls2"):
                v = 0.7 + torch.randn(shape, generator=g, device=dev) * 0.2
            elif name.endswith("a2.b"):
                v = 1.0 + torch.randn(shape, generator=g, device=dev)
            elif len(shape) == 2:
                v = torch.randn(shape, generator=g, device=dev) * (scale / shape[1] ** 0.5)
            elif "norm" in name:
                v = 1.0 + torch.randn(shape, generator=g, device=dev) * 0.1
            else:
                v = torch.randn(shape, generator=g, device=dev) * 0.1
            t[name] = v.to(torch.bfloat16)
        return self.load_weights(t)

    def load_weights(self, tensors: Dict[str, torch.Tensor]) -> "BivizenForCausalLM":
        """tensors: checkpoint name -> tensor ([out, in] linear weights).  Sizes are checked against the
        config; the fused device layouts and the frequency tables are built here."""
        cfg, dev, dt = self.config, self.device, self.dtype
        want = cfg.tensor_shapes()
        missing = [n for n in want if n not in tensors]
        if missing:
            raise KeyError(f"checkpoint lacks {missing[:4]}{'...' if len(missing) > 4 else ''}")
        for n, shape in want.items():
            got = tuple(tensors[n].shape)
            if len(got) != len(shape) or any(b >= 0 and a != b for a, b in zip(got, shape)):
                raise ValueError(f"{n}: checkpoint shape {got} != config shape {shape}")

        def w(name):  # compute-dtype copy
            return tensors[name].to(device=dev, dtype=dt).contiguous()

        def f32(name):
            return tensors[name].to(device=dev, dtype=torch.float32).contiguous()

        self.weights = {n: tensors[n] for n in want}
        self.embed, self.head, self.final_norm = w("embed"), w("head"), f32("final.norm")
        self.layers = []
        for i, lc in enumerate(cfg.layers):
            p, q, L = f"l{i}.", f"l{i}.mix.", _Layer()
            L.cfg, L.index = lc, i
            L.norm1, L.ls1, L.o = f32(p + "norm1"), f32(p + "ls1"), w(q + "o")
            if lc.type == "attention":
                # q | k | v | output gate in one projection; the gate has no bias
                L.in_w, L.in_off = stack_rows([("qkv", torch.cat([w(q + "q"), w(q + "k"), w(q + "v")])), ("g", w(q + "g"))])
                bias = torch.cat([w(q + "q.b"), w(q + "k.b"), w(q + "v.b")])
                L.in_b = torch.zeros(L.in_w.shape[0], device=dev, dtype=dt)
                L.in_b[:bias.numel()] = bias
                L.inv_freq = torch.tensor(lc.rot.frequencies(), dtype=torch.float64, device=dev) if lc.rot.dims else None
                L.v_mix = float(tensors[q + "vmix"]) if lc.v_mix else 0.0
            elif lc.type == "delta":
                L.in_w, L.in_off = stack_rows([("qkv", torch.cat([w(q + "q"), w(q + "k"), w(q + "v")])), ("g", w(q + "g")),
                                               ("a", w(q + "a")), ("b", w(q + "b"))])
                L.conv = torch.cat([f32(q + "q.conv"), f32(q + "k.conv"), f32(q + "v.conv")]).contiguous()
                L.A_log, L.dt_bias, L.norm = f32(q + "A_log"), f32(q + "dt_bias"), f32(q + "norm")
            else:
                rank = tensors[q + "a1"].shape[0]
                if tensors[q + "a2"].shape[1] != rank:
                    raise ValueError(f"{q}a2: {tensors[q + 'a2'].shape[1]} columns for a rank of {rank}")
                L.in_w, L.in_off = stack_rows([(n, w(q + n)) for n in ("q", "k", "v", "g", "a1")])
                L.a2, _ = stack_rows([("a2", w(q + "a2"))])
                L.a2_b, L.norm = f32(q + "a2.b"), f32(q + "norm")
            if lc.ff:
                L.gu = torch.empty(2 * lc.ff, cfg.width, device=dev, dtype=dt)   # rows gate_0, up_0, gate_1, ...
                L.gu[0::2], L.gu[1::2] = w(p + "mlp.gate"), w(p + "mlp.up")
                L.down, L.ls2 = w(p + "mlp.down"), f32(p + "ls2")
            self.layers.append(L)
        return self

    def state_dict(self) -> Dict[str, torch.Tensor]:
        return dict(self.weights)

    def save_pretrained(self, model_dir) -> None:
        from safetensors.torch import save_file
        d = Path(model_dir)
        d.mkdir(parents=True, exist_ok=True)
        (d / "config.json").write_text(json.dumps(self.config.to_dict(), indent=1))
        save_file({k: v.detach().cpu().contiguous() for k, v in self.weights.items()}, str(d / "model.safetensors"))

    # ---- cache geometry (read by serving.HybridCache) ----------------------------------------------
    def latent_widths(self) -> Dict[int, int]:
        """attention layer -> width of its paged per-token row: k (kv_heads * dim) | v (kv_heads * vdim)"""
        return {i: lc.kv_heads * (lc.dim + lc.vdim) for i, lc in enumerate(self.config.layers) if lc.type == "attention"}

    def state_shapes(self) -> Dict[Tuple[int, str], tuple]:
        """(layer, "scan") -> [heads, vdim, dim], the recurrent state; (layer, "conv") -> (taps - 1, channels), the last
        inputs of a delta layer's convolutions over q | k | v"""
        out = {}
        for i, lc in enumerate(self.config.layers):
            if lc.type == "attention":
                continue
            out[(i, "scan")] = (lc.heads, lc.vdim, lc.dim)
            if lc.type == "delta" and lc.conv > 1:
                out[(i, "conv")] = (lc.conv - 1, 2 * lc.kv_heads * lc.dim + lc.heads * lc.vdim)
        return out

    # ---- compute --------------------------------------------------------------------------------------
    @staticmethod
    def _part(P: torch.Tensor, L: _Layer, name: str) -> torch.Tensor:
        a, n = L.in_off[name]
        return P[:, a:a + n]

    def _attention(self, L: _Layer, h, batch, cache, v_first):
        """-> (mixer output, the values later mixing layers mix into theirs)"""
        lc = L.cfg
        pool = cache.latent[L.index]
        P = ops.linear_any(h, L.in_w, bias=L.in_b)
        qkv = self._part(P, L, "qkv")
        q = ops.rope_append(qkv, batch.positions, batch.cache_rows, pool, heads=lc.heads, kv_heads=lc.kv_heads, dim=lc.dim,
                            vdim=lc.vdim, inv_freq=L.inv_freq, unit_norm=False, eps=0.0, halves=True,
                            v_first=v_first if lc.v_mix else None, v_mix=L.v_mix)
        if lc.v_mix and v_first is None:
            v_first = qkv[:, (lc.heads + lc.kv_heads) * lc.dim:]
        o = torch.empty(h.shape[0], lc.heads * lc.vdim, dtype=self.dtype, device=self.device)
        kw = dict(heads=lc.heads, kv_heads=lc.kv_heads, dim=lc.dim, vdim=lc.vdim, page=cache.page, scale=lc.scale,
                  softcap=lc.softcap, gate=self._part(P, L, "g"), out=o)
        if batch.tiles is not None:
            ops.paged_attention(q, pool, cache.page_tables, batch.tiles, max_rows=16, **kw)
        if batch.decode_tiles is not None:
            ops.paged_attention(q, pool, cache.page_tables, batch.decode_tiles, max_rows=1, nsplit=cache.decode_splits, **kw)
        return ops.linear_any(o, L.o), v_first

    def _read_out(self, L: _Layer, o, P):
        on = ops.gated_head_norm_rows(o, L.norm, self._part(P, L, "g"), heads=L.cfg.heads, eps=self.config.norm_eps,
                                      out_dtype=self.dtype)
        return ops.linear_any(on, L.o)

    def _delta(self, L: _Layer, h, batch, cache):
        lc = L.cfg
        P = ops.linear_any(h, L.in_w)                                    # q | k | v | gate | decay | step size
        qkv = ops.causal_conv_rows(self._part(P, L, "qkv"), L.conv, None, cache.state.get((L.index, "conv")), batch.seqs,
                                   batch.row_seq, act=ops.CONV_SILU, out_dtype=self.dtype)
        o = ops.delta_scan(qkv, self._part(P, L, "a"), self._part(P, L, "b"), cache.state[(L.index, "scan")], batch.seqs,
                           heads=lc.heads, kv_heads=lc.kv_heads, dim=lc.dim, vdim=lc.vdim, A_log=L.A_log, dt_bias=L.dt_bias,
                           q_scale=lc.dim ** -0.5, unit_eps=UNIT_EPS)
        return self._read_out(L, o, P)

    def _gla(self, L: _Layer, h, batch, cache):
        lc = L.cfg
        P = ops.linear_any(h, L.in_w)                                    # q | k | v | gate | low-rank decay
        z = ops.linear_any(self._part(P, L, "a1"), L.a2)
        o = ops.gla_scan(self._part(P, L, "q"), self._part(P, L, "k"), self._part(P, L, "v"), z[:, :lc.heads * lc.dim],
                         cache.state[(L.index, "scan")], batch.seqs, heads=lc.heads, dim=lc.dim, vdim=lc.vdim,
                         q_scale=lc.dim ** -0.5, tau=lc.tau, z_bias=L.a2_b)
        return self._read_out(L, o, P)

    def _feed_forward(self, L: _Layer, h):
        return ops.linear_any(ops.linear_any(h, L.gu, glu_clamp=(GLU_ALPHA, L.cfg.limit)), L.down)

    @torch.inference_mode()
    def forward_step(self, batch, cache, layer_outputs: Optional[list] = None) -> torch.Tensor:
        """Run the rows of `batch` through all layers on top of what `cache` holds; k | v rows, convolution tails and
        recurrent states of the batch are written to the cache.  -> residual stream fp32 [T, width]."""
        eps, n = self.config.norm_eps, len(self.layers)
        x = ops.embed_rows(self.embed, batch.ids)
        h = ops.rmsnorm_rows(x, self.layers[0].norm1, eps, out_dtype=self.dtype) if n else None
        v_first = None
        for i, L in enumerate(self.layers):
            if L.cfg.type == "attention":
                y, v_first = self._attention(L, h, batch, cache, v_first)
            else:
                y = (self._delta if L.cfg.type == "delta" else self._gla)(L, h, batch, cache)
            f = self._feed_forward(L, h) if L.cfg.ff else None
            h = ops.scaled_residual_norm_rows(x, y, L.ls1, f, L.ls2 if L.cfg.ff else None,
                                              self.layers[i + 1].norm1 if i + 1 < n else None, eps, out_dtype=self.dtype)
            if layer_outputs is not None:
                layer_outputs.append(x.clone())
        return x

    @torch.inference_mode()
    def logits(self, hidden_rows: torch.Tensor) -> torch.Tensor:
        """final norm + output head for the given residual rows fp32 [n, width] -> fp32 [n, vocab]"""
        h = ops.rmsnorm_rows(hidden_rows.contiguous(), self.final_norm, self.config.norm_eps, out_dtype=self.dtype)
        return ops.glinear(h, self.head, out_dtype=torch.float32)

    @torch.inference_mode()
    def generate(self, input_ids, max_new_tokens: int = 20, eos_token_id=None, do_sample: bool = False,
                 temperature: float = 1.0, top_k: int = 0, top_p: float = 1.0, seed: Optional[int] = None,
                 slots: int = 4, **engine_kw) -> List[List[int]]:
        """input_ids: one prompt (list of ids) or a list of prompts -> new ids per prompt, through the
        continuous-batching scheduler (vila_b200.serving.generate_tokens)."""
        from ..serving import generate_tokens
        prompts = [list(map(int, input_ids))] if input_ids and not isinstance(input_ids[0], (list, tuple)) \
            else [list(map(int, p)) for p in input_ids]
        eos = [] if eos_token_id is None else ([eos_token_id] if isinstance(eos_token_id, int) else list(eos_token_id))
        return generate_tokens(self, prompts, max_new_tokens, eos, slots=slots, sample=do_sample,
                               temperature=temperature, top_k=top_k, top_p=top_p, seed=seed, **engine_kw)
