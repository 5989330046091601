"""Decoders whose layers mix tokens in different ways (recurrent state, softmax attention), listed layer by layer in config.json. The
residual stream is fp32; a layer normalises the OUTPUT of each sublayer and adds it:

    x = embed[token] * scale
    x <- x + m * norm1(mixer(x)) ;  x <- x + m * norm2(mlp(x))        for every layer (a layer without an mlp stops after the mixer)
    logits = head norm(x)

The same step serves a whole prompt, a portion of one and a single token (`forward`); one-token steps are captured in a CUDA graph over
the sequence's own state tensors, the position being read from device memory.
"""
from __future__ import annotations

from dataclasses import dataclass

import torch

import mixers as M
import plz_native as P
import seq_ops as S
from seq_state import SequenceState


@dataclass
class HybridDesign:
    """What a family of models fixes (the rest is in config.json)."""
    norm_offset: float = 0.0      # norms multiply by (norm_offset + w)


@dataclass
class LayerSpec:
    type: str
    mixer: dict
    mlp: dict | None


@dataclass
class HybridConfig:
    width: int
    vocab: int
    layers: list
    eps: float
    embed_scale: float = 1.0
    residual_mult: float = 1.0

    @classmethod
    def from_dict(cls, c: dict) -> "HybridConfig":
        layers = []
        for i, e in enumerate(c["layers"]):
            if e["type"] not in M.MIXERS:
                raise ValueError(f"layer {i}: unknown mixer {e['type']!r}")
            mlp = e.get("mlp")
            if mlp is not None and mlp["kind"] not in M.MLPS:
                raise ValueError(f"layer {i}: unknown feed-forward {mlp['kind']!r}")
            layers.append(LayerSpec(e["type"], dict(e["mixer"]), dict(mlp) if mlp is not None else None))
        return cls(c["width"], c["vocab"], layers, c["norm"]["eps"], c["embedding"]["scale"], c["residual_mult"])


def tensor_shapes(config: dict) -> dict:
    """Stored name -> shape of every tensor of a model with this config.json (ranks and table sizes that only the tensors give take
    their defaults)."""
    w, out = config["width"], {"embed": (config["vocab"], config["width"])}
    for i, e in enumerate(config["layers"]):
        out[f"l{i}.norm1"] = (w,)
        out.update({f"l{i}.mix.{k}": s for k, s in M.MIXERS[e["type"]].shapes(e["mixer"], w).items()})
        if e.get("mlp") is not None:
            out[f"l{i}.norm2"] = (w,)
            out.update({f"l{i}.mlp.{k}": s for k, s in M.MLPS[e["mlp"]["kind"]].shapes(e["mlp"], w).items()})
    out["final.norm"] = (w,)
    out["head"] = (config["vocab"], w)
    return out


def random_tensors(config: dict, seed: int = 0, device="cpu") -> dict:
    """Synthetic bf16 weights: matrices N(0, 1 / columns), plain norm weights 1 + N(0, 0.1^2), everything else N(0, 0.3^2)."""
    g = torch.Generator(device=device).manual_seed(seed)
    out = {}
    for name, shape in tensor_shapes(config).items():
        t = torch.randn(shape, generator=g, device=device)
        if name in ("embed",):
            pass
        elif name.endswith((".mix.norm", ".q.norm", ".k.norm")):
            t = 1.0 + 0.1 * t
        elif len(shape) == 2 and not name.endswith((".rel", ".conv")):
            t = t * shape[1] ** -0.5
        else:
            t = t * 0.3
        out[name] = t.to(torch.bfloat16)
    return out


class _Layer:
    def __init__(self, spec: LayerSpec, tensors, prefix: str, width: int, dtype, device):
        L = M.Loader(tensors, prefix, dtype, device)
        self.mixer = M.MIXERS[spec.type](spec.mixer, M.Loader(tensors, prefix + "mix.", dtype, device), width)
        self.norm1 = L.f32("norm1", (width,))
        self.mlp = self.norm2 = None
        if spec.mlp is not None:
            self.mlp = M.MLPS[spec.mlp["kind"]](spec.mlp, M.Loader(tensors, prefix + "mlp.", dtype, device), width)
            self.norm2 = L.f32("norm2", (width,))


class HybridModel:
    DESIGN = HybridDesign()
    DTYPES = (torch.bfloat16, torch.float32)

    def __init__(self, cfg: HybridConfig, tensors, dtype: torch.dtype = torch.bfloat16, device="cuda"):
        """tensors: mapping of stored name -> CPU tensor (safetensors_io.SafeTensors or a dict)."""
        if dtype not in self.DTYPES:
            raise ValueError(f"{dtype} is not supported")
        self.cfg, self.dtype, self.device = cfg, dtype, torch.device(device)
        top = M.Loader(tensors, "", dtype, self.device)
        self.embed = top.mat("embed", (cfg.vocab, cfg.width))
        self.head = top.mat("head", (cfg.vocab, cfg.width))
        self.final_norm = top.f32("final.norm", (cfg.width,))
        self.layers = [_Layer(s, tensors, f"l{i}.", cfg.width, dtype, self.device) for i, s in enumerate(cfg.layers)]
        self.use_graph = True

    @classmethod
    def from_config(cls, config: dict, tensors, dtype=torch.bfloat16, device="cuda"):
        return cls(HybridConfig.from_dict(config), tensors, dtype, device)

    @classmethod
    def random(cls, config: dict, device="cuda", seed: int = 0, dtype=torch.bfloat16):
        return cls.from_config(config, random_tensors(config, seed, device), dtype, device)

    @property
    def vocab(self) -> int:
        return self.cfg.vocab

    def weight_bytes(self) -> int:
        """Bytes of the matrices a decode step reads (embedding table aside)."""
        seen = [self.head]
        for l in self.layers:
            seen += [t for m in (l.mixer, l.mlp) if m is not None for t in vars(m).values() if isinstance(t, torch.Tensor) and t.dim() == 2 and t.dtype == self.dtype]
        return sum(t.numel() * t.element_size() for t in seen)

    def new_cache(self, B: int, T_max: int) -> SequenceState:
        return SequenceState([l.mixer.state_spec() for l in self.layers], B, T_max, self.dtype, self.device)

    # ---- one step ------------------------------------------------------------------------------------------------
    def hidden(self, ids: torch.Tensor, cache: SequenceState, host_pos: int, layers_out=None) -> torch.Tensor:
        """Residual stream fp32 [B * n, width] after all layers for ids int64 [B, n]; advances cache.pos on the device only."""
        c, off = self.cfg, self.DESIGN.norm_offset
        B, n = ids.shape
        ctx = M.StepContext(B, n, cache.pos, host_pos, c.eps)
        x, xb = S.embed(self.embed, ids, c.embed_scale)
        for layer, st in zip(self.layers, cache.layers):
            S.residual_norm(layer.mixer.forward(xb, st, ctx), layer.norm1, off, c.residual_mult, c.eps, x, xb)
            if layer.mlp is not None:
                S.residual_norm(layer.mlp.forward(xb), layer.norm2, off, c.residual_mult, c.eps, x, xb)
            if layers_out is not None:
                layers_out.append(x.clone())
        S.advance(cache.pos, n)
        return x

    def logits(self, x: torch.Tensor, rows=None) -> torch.Tensor:
        """fp32 logits of the given rows (int64 device tensor; None: all) of the residual stream."""
        h = S.rows_norm(x, rows, self.final_norm, self.DESIGN.norm_offset, self.cfg.eps, self.dtype)
        return S.linear(h, self.head, out_f32=True) if h.shape[0] <= 16 else S.linear(h, self.head).float()

    def forward(self, ids: torch.Tensor, cache: SequenceState, want=None):
        """Run ids int64 [B, n] from the state in `cache`; want: rows (b * n + t) whose logits are returned, fp32 [len(want), vocab]
        (None when nothing is wanted)."""
        B, n = ids.shape
        if B != cache.B:
            raise ValueError(f"{B} sequences for a state of {cache.B}")
        if n == 0:
            return None
        if cache.length + n > cache.capacity:
            raise ValueError(f"{cache.length} + {n} tokens exceed the capacity {cache.capacity} of the state")
        if n == 1 and self.use_graph:
            out = self._token(ids, cache)
            cache.length += 1
            if want is None or len(want) == 0:
                return None
            return out.clone() if list(want) == list(range(B)) else out[torch.as_tensor(want, device=self.device)]
        ids = ids.to(self.device).contiguous()
        x = self.hidden(ids, cache, cache.length)
        cache.length += n
        if want is None or len(want) == 0:
            return None
        return self.logits(x, torch.as_tensor(want, dtype=torch.int64, device=self.device))

    def _token(self, ids: torch.Tensor, cache: SequenceState) -> torch.Tensor:
        """One token per sequence. The first such step of a state runs eagerly, the second is captured (capturing runs nothing) and from
        then on replayed."""
        g = cache.step_graph
        if g is None:
            cache.step_graph = (None, torch.empty(cache.B, 1, dtype=torch.int64, device=self.device), None)
            cache.step_graph[1].copy_(ids)
            return self._token_chain(cache.step_graph[1], cache)
        graph, buf, out = g
        if graph is None:
            graph = torch.cuda.CUDAGraph()
            torch.cuda.synchronize()
            with torch.cuda.graph(graph):
                out = self._token_chain(buf, cache)
            cache.step_graph = (graph, buf, out)
        buf.copy_(ids)
        graph.replay()
        return out

    def _token_chain(self, ids: torch.Tensor, cache: SequenceState) -> torch.Tensor:
        lib = P.lib()
        lib.plz_set_smallm_overlap(1)        # kernels of the chain may start under their predecessors (programmatic dependent launch)
        try:
            return self.logits(self.hidden(ids, cache, -1))
        finally:
            lib.plz_set_smallm_overlap(0)

    # ---- the calls PalettizedQwen has -----------------------------------------------------------------------------
    def prefill(self, ids: torch.Tensor, cache: SequenceState, want_logits: bool = True):
        """ids int64 [B, S]; logits of the last position of every sequence (or None)."""
        B, n = ids.shape
        return self.forward(ids, cache, [b * n + n - 1 for b in range(B)] if want_logits else None)

    def decode_step(self, ids: torch.Tensor, cache: SequenceState) -> torch.Tensor:
        """Logits fp32 [B, vocab] after ids (int64 [B])."""
        return self.forward(ids.view(-1, 1), cache, list(range(ids.numel())))


class Gopunex(HybridModel):
    """Lightning, channel-wise gated delta and distance-bias attention layers in any order; norm weights stored around zero."""
    DESIGN = HybridDesign(norm_offset=1.0)
