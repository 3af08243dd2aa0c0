"""Nibelix: a decoder-only language model of lightning attention and windowed differential attention with parallel
sublayers, Dynamic Tanh norms and routed experts on the ragged-batch kernels.

Residual stream x (fp32).  Layer i:  x += m * (ls1 * mixer(N1(x)) + ls2 * ff(N2(x))), both sublayers read the same x
through a norm of their own, N(x) = tanh(alpha x) * w + b; ls1 / ls2 are per-channel scales, m = `residual_mult`; a layer
may have no feed-forward.  Mixers (config `layers[i].type`):

  lightning   q, k, v = SiLU of their projections; per head S <- decay S + k v^T, o = S^T q with a constant decay per head;
              all heads together RMS-normed (weight per channel), times sigmoid of a gate projection
  attention   differential attention: every query / key head is two maps over the same values, each a softmax over the
              last `mask.size` positions with rotary positions (halves layout) on the first `rot.dims` columns of each map;
              a1 - lambda a2, RMS-normed per head, times (1 - diff), times a sigmoid gate per head; lambda =
              exp(lq1 . lk1) - exp(lq2 . lk2) + diff

Feed-forwards (`mlp.kind`): dense  down(gelu_tanh(gate h) * up h);  moe  softmax router over experts and identity experts
(whose output is h itself), a correction added for the choice only, groups ranked by their best choice value, weights the
plain scores times `router.scale`; experts down(gelu(up h)); a shared expert of the same form times sigmoid(w_sg . h).
Logits: final norm, head, softcap * tanh(z / softcap).

One step takes a RaggedBatch and a HybridCache owned by the serving engine (vila_b200/serving.py): attention layers keep
k (both maps) | v rows in a paged pool, lightning layers their state in the sequence's slot.  dtype bfloat16: projections on
the tcgen05 GEMM (shapes it does not take go to the CUDA-core grouped kernel); positions and angles, norms, scores and
softmax, the maps' combination, routers, states with everything that enters them, and the residual sum in fp32.  dtype
float32: the same kernels with fp32 tensors and the CUDA-core linear layer throughout.
"""
from __future__ import annotations

import json
import math
from dataclasses import dataclass, field
from pathlib import Path
from typing import Dict, List, Optional, Tuple

import torch

from .. import ops
from .ludazen import RotaryConfig
from .moronex import read_safetensors, stack_rows

ARCHITECTURE = "Nibelix"


@dataclass
class NibelixLayerConfig:
    type: str                         # "lightning" | "attention"
    heads: int
    dim: int
    vdim: int
    decay: List[float] = field(default_factory=list)   # lightning: one per head
    kv_heads: int = 0                 # attention
    scale: float = 1.0
    diff: float = 0.0
    window: int = 0                   # mask.size; 0: every earlier position is seen
    rot: Optional[RotaryConfig] = None
    mlp_kind: Optional[str] = None    # "dense" | "moe" | None
    ff: int = 0                       # dense: hidden size; moe: hidden size of one expert
    experts: int = 0
    identity: int = 0                 # router outputs after the experts whose "expert" is the input itself
    top: int = 0
    groups: int = 1
    keep: int = 1
    router_scale: float = 1.0
    shared_ff: int = 0                # 0: no shared expert

    @property
    def outputs(self) -> int:
        return self.experts + self.identity


@dataclass
class NibelixConfig:
    vocab: int
    width: int
    norm_eps: float
    residual_mult: float = 1.0
    logit_softcap: float = 0.0        # 0: logits are not capped
    layers: List[NibelixLayerConfig] = field(default_factory=list)
    architecture: str = ARCHITECTURE

    @staticmethod
    def from_dict(d: dict) -> "NibelixConfig":
        layers = []
        for i, spec in enumerate(d["layers"]):
            m, kind = spec["mixer"], spec["type"]
            lc = NibelixLayerConfig(type=kind, heads=int(m["heads"]), dim=int(m["dim"]), vdim=int(m["vdim"]))
            if kind == "lightning":
                lc.decay = [float(v) for v in m["decay"]]
            elif kind == "attention":
                lc.kv_heads, lc.scale, lc.diff = int(m["kv_heads"]), float(m["scale"]), float(m["diff"])
                lc.window = int(m["mask"]["size"]) if m.get("mask") else 0
                lc.rot = RotaryConfig.from_dict(m["rot"]) if m.get("rot") else RotaryConfig(dims=0, base=1.0)
            else:
                raise ValueError(f"layer {i}: unknown mixer type {kind!r}")
            mlp = spec.get("mlp")
            if mlp is not None:
                lc.mlp_kind = mlp["kind"]
                if lc.mlp_kind == "dense":
                    lc.ff = int(mlp["ff"])
                elif lc.mlp_kind == "moe":
                    r, g = mlp["router"], mlp["router"].get("groups") or {}
                    lc.ff, lc.experts, lc.top = int(mlp["expert"]["ff"]), int(r["experts"]), int(r["top"])
                    lc.identity, lc.router_scale = int(r.get("identity") or 0), float(r.get("scale", 1.0))
                    lc.groups, lc.keep = int(g.get("count", 1)), int(g.get("keep", 1))
                    lc.shared_ff = int(mlp["shared"]["ff"]) if mlp.get("shared") else 0
                else:
                    raise ValueError(f"layer {i}: unknown feed-forward kind {lc.mlp_kind!r}")
            layers.append(lc)
        cfg = NibelixConfig(vocab=int(d["vocab"]), width=int(d["width"]), norm_eps=float(d["norm"]["eps"]),
                            residual_mult=float(d.get("residual_mult", 1.0)),
                            logit_softcap=float(d.get("logit_softcap") or 0.0), layers=layers)
        cfg.validate()
        return cfg

    def validate(self) -> None:
        if self.logit_softcap < 0:
            raise ValueError(f"logit_softcap {self.logit_softcap}")
        for i, lc in enumerate(self.layers):
            if lc.heads < 1 or lc.dim < 1 or lc.vdim < 1:
                raise ValueError(f"layer {i}: heads {lc.heads}, dim {lc.dim}, vdim {lc.vdim}")
            if lc.type == "lightning":
                if len(lc.decay) != lc.heads:
                    raise ValueError(f"layer {i}: {len(lc.decay)} decays for {lc.heads} heads")
                if lc.dim > 512:
                    raise ValueError(f"layer {i}: a recurrent state of dim {lc.dim} (at most 512)")
            else:
                if lc.kv_heads < 1 or lc.heads % lc.kv_heads:
                    raise ValueError(f"layer {i}: heads {lc.heads} / kv_heads {lc.kv_heads}")
                if lc.rot.dims % 2 or lc.rot.dims > lc.dim or lc.window < 0:
                    raise ValueError(f"layer {i}: rot.dims {lc.rot.dims} of {lc.dim}, mask.size {lc.window}")
            if lc.mlp_kind is not None and lc.ff < 1:
                raise ValueError(f"layer {i}: feed-forward size {lc.ff}")
            if lc.mlp_kind == "moe":
                if lc.experts < 1 or lc.identity < 0 or lc.groups < 1 or lc.outputs % lc.groups:
                    raise ValueError(f"layer {i}: {lc.experts} + {lc.identity} experts in {lc.groups} groups")
                if not 1 <= lc.keep <= lc.groups or not 1 <= lc.top <= lc.keep * (lc.outputs // lc.groups):
                    raise ValueError(f"layer {i}: router top {lc.top} of {lc.keep} of {lc.groups} groups")

    def to_dict(self) -> dict:
        out = []
        for lc in self.layers:
            m = {"dim": lc.dim, "heads": lc.heads, "vdim": lc.vdim}
            if lc.type == "lightning":
                m.update(decay=list(lc.decay))
            else:
                m.update(diff=lc.diff, kv_heads=lc.kv_heads, rot=lc.rot.to_dict(), scale=lc.scale)
                if lc.window:
                    m["mask"] = {"size": lc.window}
            mlp = None
            if lc.mlp_kind == "dense":
                mlp = {"ff": lc.ff, "kind": "dense"}
            elif lc.mlp_kind == "moe":
                mlp = {"expert": {"ff": lc.ff}, "kind": "moe",
                       "router": {"experts": lc.experts, "groups": {"count": lc.groups, "keep": lc.keep},
                                  "identity": lc.identity, "scale": lc.router_scale, "top": lc.top}}
                if lc.shared_ff:
                    mlp["shared"] = {"ff": lc.shared_ff}
            out.append({"mixer": m, "mlp": mlp, "type": lc.type})
        return {"architecture": self.architecture, "layers": out, "logit_softcap": self.logit_softcap,
                "norm": {"eps": self.norm_eps}, "residual_mult": self.residual_mult, "vocab": self.vocab, "width": self.width}

    def tensor_shapes(self) -> Dict[str, tuple]:
        """name -> shape of every checkpoint tensor (the layout `load_weights` expects)."""
        W, s = self.width, {}

        def norm(name):
            s[name], s[name + ".b"], s[name + ".alpha"] = (W,), (W,), ()
        s["embed"] = (self.vocab, W)
        for i, lc in enumerate(self.layers):
            p, q, f = f"l{i}.", f"l{i}.mix.", f"l{i}.mlp."
            norm(p + "norm1")
            s[p + "ls1"] = (W,)
            if lc.type == "lightning":
                hd, hv = lc.heads * lc.dim, lc.heads * lc.vdim
                s[q + "q"], s[q + "k"], s[q + "v"], s[q + "g"] = (hd, W), (hd, W), (hv, W), (hv, W)
                s[q + "norm"] = (hv,)
            else:
                s[q + "q"], s[q + "k"] = (2 * lc.heads * lc.dim, W), (2 * lc.kv_heads * lc.dim, W)
                s[q + "v"], s[q + "g"] = (lc.kv_heads * lc.vdim, W), (lc.heads, W)
                for n in ("lq1", "lk1", "lq2", "lk2"):
                    s[q + n] = (lc.dim,)
            s[q + "o"] = (W, lc.heads * lc.vdim)
            if lc.mlp_kind is not None:
                norm(p + "norm2")
                s[p + "ls2"] = (W,)
            if lc.mlp_kind == "dense":
                s[f + "gate"], s[f + "up"], s[f + "down"] = (lc.ff, W), (lc.ff, W), (W, lc.ff)
            elif lc.mlp_kind == "moe":
                for e in range(lc.experts):
                    s[f + f"e{e}.up"], s[f + f"e{e}.down"] = (lc.ff, W), (W, lc.ff)
                s[f + "router"], s[f + "correction"] = (lc.outputs, W), (lc.outputs,)
                if lc.shared_ff:
                    s[f + "shared.up"], s[f + "shared.down"] = (lc.shared_ff, W), (W, lc.shared_ff)
                    s[f + "shared.sg"] = (1, W)
        norm("final.norm")
        s["head"] = (self.vocab, W)
        return s


class _Layer:
    """Device tensors of one layer in the layout the kernels want."""


class NibelixForCausalLM:
    """Weights + the per-step compute of the architecture.  Sequences, pages, state slots, batching and
    sampling belong to `vila_b200.serving.TokenEngine`, which calls `forward_step` / `logits`."""

    def __init__(self, cfg: NibelixConfig, device="cuda", dtype=torch.bfloat16):
        assert dtype in (torch.bfloat16, torch.float32)
        cfg.validate()
        self.config, self.device, self.dtype = cfg, torch.device(device), dtype
        self.vocab_size = cfg.vocab
        self.weights: Dict[str, torch.Tensor] = {}
        self.layers: List[_Layer] = []

    # ---- weights ----------------------------------------------------------------------------------
    @classmethod
    def from_pretrained(cls, model_dir, device="cuda", dtype=torch.bfloat16) -> "NibelixForCausalLM":
        d = Path(model_dir)
        cfg = NibelixConfig.from_dict(json.loads((d / "config.json").read_text()))
        files = sorted(d.glob("*.safetensors"))
        if not files:
            raise FileNotFoundError(f"no *.safetensors under {d}")
        tensors: Dict[str, torch.Tensor] = {}
        for f in files:
            tensors.update(read_safetensors(f))
        return cls(cfg, device, dtype).load_weights(tensors)

    def init_random(self, seed: int = 0, scale: float = 1.0, on_device: bool = False) -> "NibelixForCausalLM":
        """Random bf16-representable weights.  on_device: draw them on the model's device (large models)."""
        dev = self.device if on_device else torch.device("cpu")
        g = torch.Generator(device=dev).manual_seed(seed)
        t = {}
        for name, shape in self.config.tensor_shapes().items():
            last = name.rsplit(".", 1)[-1]
            if last == "alpha":
                v = 0.5 + 0.5 * torch.rand(shape, generator=g, device=dev)
            elif last in ("ls1", "ls2"):
                v = 0.7 + torch.randn(shape, generator=g, device=dev) * 0.2
            elif last in ("lq1", "lk1", "lq2", "lk2"):
                v = torch.randn(shape, generator=g, device=dev) * 0.2
            elif last == "correction":
                v = torch.randn(shape, generator=g, device=dev) * 0.2
            elif len(shape) == 2:
                v = torch.randn(shape, generator=g, device=dev) * (scale / shape[1] ** 0.5)
            elif last == "b":
                v = torch.randn(shape, generator=g, device=dev) * 0.1
            else:   # norm weights
                v = 1.0 + torch.randn(shape, generator=g, device=dev) * 0.1
            t[name] = v.to(torch.bfloat16)
        return self.load_weights(t)

    def load_weights(self, tensors: Dict[str, torch.Tensor]) -> "NibelixForCausalLM":
        """tensors: checkpoint name -> tensor ([out, in] linear weights).  Sizes are checked against the
        config; the fused device layouts, the frequency tables and each layer's lambda are built here."""
        cfg, dev, dt = self.config, self.device, self.dtype
        want = cfg.tensor_shapes()
        missing = [n for n in want if n not in tensors]
        if missing:
            raise KeyError(f"checkpoint lacks {missing[:4]}{'...' if len(missing) > 4 else ''}")
        for n, shape in want.items():
            if tuple(tensors[n].shape) != tuple(shape):
                raise ValueError(f"{n}: checkpoint shape {tuple(tensors[n].shape)} != config shape {shape}")

        def w(name):  # compute-dtype copy
            return tensors[name].to(device=dev, dtype=dt).contiguous()

        def f32(name):
            return tensors[name].to(device=dev, dtype=torch.float32).contiguous()

        def norm(name):
            return ops.TanhNorm(float(tensors[name + ".alpha"]), f32(name), f32(name + ".b"))

        def dot(a, b):
            return float((tensors[a].double() * tensors[b].double()).sum())

        self.weights = {n: tensors[n] for n in want}
        self.embed, self.head, self.final_norm = w("embed"), w("head"), norm("final.norm")
        self.layers = []
        for i, lc in enumerate(cfg.layers):
            p, q, f, L = f"l{i}.", f"l{i}.mix.", f"l{i}.mlp.", _Layer()
            L.cfg, L.index = lc, i
            L.norms, L.ls1, L.o = [norm(p + "norm1")], f32(p + "ls1"), w(q + "o")
            if lc.type == "lightning":
                L.in_w, L.in_off = stack_rows([(n, w(q + n)) for n in ("q", "k", "v", "g")])
                L.decay = torch.tensor(lc.decay, dtype=torch.float32, device=dev)
                L.norm = f32(q + "norm")
            else:
                L.in_w, L.in_off = stack_rows([("qkv", torch.cat([w(q + "q"), w(q + "k"), w(q + "v")])), ("g", w(q + "g"))])
                L.inv_freq = torch.tensor(lc.rot.frequencies(), dtype=torch.float64, device=dev) if lc.rot.dims else None
                lam = math.exp(dot(q + "lq1", q + "lk1")) - math.exp(dot(q + "lq2", q + "lk2")) + lc.diff
                L.diff = (lam, 1.0 - lc.diff, cfg.norm_eps)
            if lc.mlp_kind is not None:
                L.norms.append(norm(p + "norm2"))
                L.ls2 = f32(p + "ls2")
            if lc.mlp_kind == "dense":
                L.gu = torch.empty(2 * lc.ff, cfg.width, device=dev, dtype=dt)   # rows gate_0, up_0, gate_1, ...
                L.gu[0::2], L.gu[1::2] = w(f + "gate"), w(f + "up")
                L.down = w(f + "down")
            elif lc.mlp_kind == "moe":
                L.up = torch.stack([w(f + f"e{e}.up") for e in range(lc.experts)]).contiguous()
                L.down = torch.stack([w(f + f"e{e}.down") for e in range(lc.experts)]).contiguous()
                L.router, L.correction = f32(f + "router"), f32(f + "correction")
                L.shared_gate = None
                if lc.shared_ff:
                    L.shared_up, L.shared_down = w(f + "shared.up"), w(f + "shared.down")
                    L.shared_gate = f32(f + "shared.sg").view(-1)
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
        """attention layer -> width of its paged per-token row: k, two maps (kv_heads * 2 * dim) | v (kv_heads * vdim)"""
        return {i: lc.kv_heads * (2 * lc.dim + lc.vdim) for i, lc in enumerate(self.config.layers) if lc.type == "attention"}

    def state_shapes(self) -> Dict[Tuple[int, str], tuple]:
        """(lightning layer, "scan") -> [heads, vdim, dim], its recurrent state"""
        return {(i, "scan"): (lc.heads, lc.vdim, lc.dim) for i, lc in enumerate(self.config.layers) if lc.type == "lightning"}

    # ---- compute --------------------------------------------------------------------------------------
    @staticmethod
    def _part(P: torch.Tensor, L: _Layer, name: str) -> torch.Tensor:
        a, n = L.in_off[name]
        return P[:, a:a + n]

    def _lightning(self, L: _Layer, h, batch, cache):
        lc = L.cfg
        P = ops.linear_any(h, L.in_w)                                    # q | k | v | gate, before their activations
        o = ops.decay_scan(self._part(P, L, "q"), self._part(P, L, "k"), self._part(P, L, "v"), cache.state[(L.index, "scan")],
                           batch.seqs, heads=lc.heads, dim=lc.dim, vdim=lc.vdim, decay=L.decay, silu=True)
        on = ops.gated_head_norm_rows(o, L.norm, self._part(P, L, "g"), heads=1, eps=self.config.norm_eps, out_dtype=self.dtype,
                                      gate_act=ops.ACT_SIGMOID)
        return ops.linear_any(on, L.o)

    def _attention(self, L: _Layer, h, batch, cache):
        lc = L.cfg
        pool = cache.latent[L.index]
        P = ops.linear_any(h, L.in_w)                                    # q (two maps) | k (two maps) | v | gate
        q = ops.rope_append(self._part(P, L, "qkv"), batch.positions, batch.cache_rows, pool, heads=lc.heads,
                            kv_heads=lc.kv_heads, dim=lc.dim, vdim=lc.vdim, inv_freq=L.inv_freq, unit_norm=False, eps=0.0,
                            halves=True, maps=2)
        o = torch.empty(h.shape[0], lc.heads * lc.vdim, dtype=self.dtype, device=self.device)
        kw = dict(heads=lc.heads, kv_heads=lc.kv_heads, dim=lc.dim, vdim=lc.vdim, page=cache.page, scale=lc.scale,
                  window=lc.window, diff=L.diff, gate=self._part(P, L, "g"), out=o)
        if batch.tiles is not None:
            ops.paged_attention(q, pool, cache.page_tables, batch.tiles, max_rows=16, **kw)
        if batch.decode_tiles is not None:
            # one CTA per 64 keys that a row can see, at most the pool's choice
            splits = min(cache.decode_splits, (lc.window + 63) // 64) if lc.window else cache.decode_splits
            ops.paged_attention(q, pool, cache.page_tables, batch.decode_tiles, max_rows=1, nsplit=splits, **kw)
        return ops.linear_any(o, L.o)

    def _dense(self, L: _Layer, h) -> dict:
        return dict(b=ops.linear_any(ops.linear_any(h, L.gu, geglu=True), L.down))

    def _experts(self, L: _Layer, h) -> dict:
        lc, T = L.cfg, h.shape[0]
        idx, wt, gate = ops.moe_route_scores(h, L.router, L.correction, lc.top, score=ops.SCORE_SOFTMAX, groups=lc.groups,
                                             keep=lc.keep, group_top=1, scale=lc.router_scale, gate_w=L.shared_gate)
        seg, srt = ops.moe_group(idx, lc.experts)                        # identity choices belong to no segment
        act = ops.glinear(h, L.up, groups=lc.experts, seg=seg, a_rows=srt, a_row_div=lc.top, act=ops.ACT_GELU_ERF)
        parts = ops.glinear(act, L.down, groups=lc.experts, seg=seg, o_rows=srt, row_scale=wt.view(-1),
                            out_dtype=torch.float32, out_rows_total=T * lc.top)
        shared = None
        if lc.shared_ff:
            shared = ops.linear_any(ops.linear_any(h, L.shared_up, act=ops.ACT_GELU_ERF), L.shared_down)
        return dict(b=shared, b_gate=gate, part=parts, n_partials=lc.top, idx=idx, weight=wt, experts=lc.experts, h=h)

    @torch.inference_mode()
    def forward_step(self, batch, cache, layer_outputs: Optional[list] = None) -> torch.Tensor:
        """Run the rows of `batch` through all layers on top of what `cache` holds; k | v rows and recurrent states of the
        batch are written to the cache.  -> residual stream fp32 [T, width]."""
        n = len(self.layers)
        x = torch.empty(batch.T, self.config.width, dtype=torch.float32, device=self.device)
        hs = ops.tanh_residual_rows(x, self.layers[0].norms if n else [], out_dtype=self.dtype, table=self.embed, ids=batch.ids)
        for i, L in enumerate(self.layers):
            y = (self._lightning if L.cfg.type == "lightning" else self._attention)(L, hs[0], batch, cache)
            ff = {}
            if L.cfg.mlp_kind is not None:
                ff = dict((self._dense if L.cfg.mlp_kind == "dense" else self._experts)(L, hs[1]), b_scale=L.ls2)
            hs = ops.tanh_residual_rows(x, self.layers[i + 1].norms if i + 1 < n else [], out_dtype=self.dtype, a=y,
                                        a_scale=L.ls1, mult=self.config.residual_mult, **ff)
            if layer_outputs is not None:
                layer_outputs.append(x.clone())
        return x

    @torch.inference_mode()
    def logits(self, hidden_rows: torch.Tensor) -> torch.Tensor:
        """final norm + output head (+ cap) for the given residual rows fp32 [n, width] -> fp32 [n, vocab]"""
        h, = ops.tanh_residual_rows(hidden_rows.contiguous(), [self.final_norm], out_dtype=self.dtype)
        cap = self.config.logit_softcap
        if cap:
            return ops.glinear(h, self.head, out_dtype=torch.float32, act=ops.ACT_SOFTCAP, act_params=(cap, 0.0))
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
