"""Decoders whose layers mix tokens in different ways (recurrent state, softmax attention, attention over latents), listed layer by layer in
config.json. The residual stream is fp32. What a family fixes is in its HybridDesign; with norms on the outputs of the sublayers only

    x = embed[token] * scale
    x <- x + m * norm1(mixer(x)) ;  x <- x + m * norm2(mlp(x))        for every layer (a layer without an mlp stops after the mixer)
    logits = head norm(x)

and with norms on both sides x <- x + ls1 * norm1b(mixer(norm1(x))), likewise for the mlp. A run of layers may be passed through several
times with the same weights (LoopSpec); every pass has its own state.

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
    dense_mlp: str = "relu2"      # the feed-forward that config.json calls 'dense'
    pre_norm: bool = False        # sublayers read norm1 / norm2 of the stream; the norms of their outputs are norm1b / norm2b
    layer_scale: bool = False     # the normed outputs are multiplied by the vectors ls1 / ls2
    embed_norm: bool = False      # the embedding is normed (embed.norm)
    tied_head: bool = False       # logits against the embedding table


@dataclass
class LayerSpec:
    type: str
    mixer: dict
    mlp: dict | None


@dataclass
class LoopSpec:
    """Layers start .. stop - 1 run `times` times in a row. Ahead of every pass but the first the embedding is added to the stream, ahead
    of pass t the vector t of 'loop.step'."""
    start: int
    stop: int
    times: int


@dataclass
class HybridConfig:
    width: int
    vocab: int
    layers: list
    eps: float
    embed_scale: float = 1.0
    residual_mult: float = 1.0
    loop: LoopSpec | None = None

    @classmethod
    def from_dict(cls, c: dict) -> "HybridConfig":
        layers = []
        for i, e in enumerate(c["layers"]):
            if e["type"] not in M.MIXERS:
                raise ValueError(f"layer {i}: unknown mixer {e['type']!r}")
            mlp = e.get("mlp")
            if mlp is not None and mlp["kind"] != "dense":
                raise ValueError(f"layer {i}: unknown feed-forward {mlp['kind']!r}")
            layers.append(LayerSpec(e["type"], dict(e["mixer"]), dict(mlp) if mlp is not None else None))
        loop = c.get("loop")
        if loop is not None:
            loop = LoopSpec(loop["start"], loop["stop"], loop["times"])
            if not 0 <= loop.start < loop.stop <= len(layers) or loop.times < 1:
                raise ValueError(f"{loop} over {len(layers)} layers")
        return cls(c["width"], c["vocab"], layers, c["norm"]["eps"], c.get("embedding", {}).get("scale", 1.0), c.get("residual_mult", 1.0), loop)

    def runs(self):
        """[(layer, pass that starts with it or None)] in the order they run."""
        n, lp = len(self.layers), self.loop
        if lp is None:
            return [(i, None) for i in range(n)]
        body = [(i, t if i == lp.start else None) for t in range(lp.times) for i in range(lp.start, lp.stop)]
        return [(i, None) for i in range(lp.start)] + body + [(i, None) for i in range(lp.stop, n)]


def design_of(config: dict) -> HybridDesign:
    return ARCHITECTURES[config["architecture"]].DESIGN


def tensor_shapes(config: dict) -> dict:
    """Stored name -> shape of every tensor of a model with this config.json (ranks and table sizes that only the tensors give take
    their defaults)."""
    d = design_of(config)
    w, out = config["width"], {"embed": (config["vocab"], config["width"])}
    if d.embed_norm:
        out["embed.norm"] = (w,)
    if config.get("loop"):
        out["loop.step"] = (config["loop"]["times"], w)
    for i, e in enumerate(config["layers"]):
        names = ["1", "2"] if e.get("mlp") is not None else ["1"]
        for k in names:
            out[f"l{i}.norm{k}"] = (w,)
            if d.pre_norm:
                out[f"l{i}.norm{k}b"] = (w,)
            if d.layer_scale:
                out[f"l{i}.ls{k}"] = (w,)
        out.update({f"l{i}.mix.{k}": s for k, s in M.MIXERS[e["type"]].shapes(e["mixer"], w).items()})
        if e.get("mlp") is not None:
            out.update({f"l{i}.mlp.{k}": s for k, s in M.MLPS[d.dense_mlp].shapes(e["mlp"], w).items()})
    out["final.norm"] = (w,)
    if not d.tied_head:
        out["head"] = (config["vocab"], w)
    return out


def random_tensors(config: dict, seed: int = 0, device="cpu") -> dict:
    """Synthetic bf16 weights: matrices N(0, 1 / columns), plain norm weights 1 + N(0, 0.1^2), everything else N(0, 0.3^2)."""
    g = torch.Generator(device=device).manual_seed(seed)
    plain = (".mix.norm", ".q.norm", ".k.norm", ".dq.norm", ".dkv.norm")
    if design_of(config).norm_offset == 0.0:
        plain += ("embed.norm", "final.norm", ".norm1", ".norm2", ".norm1b", ".norm2b")
    out = {}
    for name, shape in tensor_shapes(config).items():
        t = torch.randn(shape, generator=g, device=device)
        if name in ("embed",):
            pass
        elif name.endswith(plain):
            t = 1.0 + 0.1 * t
        elif len(shape) == 2 and not name.endswith((".rel", ".conv", ".step")):
            t = t * shape[1] ** -0.5
        else:
            t = t * 0.3
        out[name] = t.to(torch.bfloat16)
    return out


class _Layer:
    """Mixer and feed-forward of one layer; post1 / post2 weigh the norms of their outputs (layer scales included), pre1 / pre2 those of
    their inputs (None: they read the stream itself)."""

    def __init__(self, spec: LayerSpec, design: HybridDesign, tensors, prefix: str, width: int, dtype, device):
        L = M.Loader(tensors, prefix, dtype, device)

        def norms(k):
            post = L.f32(f"norm{k}b" if design.pre_norm else f"norm{k}", (width,))
            if design.layer_scale:
                post = ((post + design.norm_offset) * L.f32(f"ls{k}", (width,)) - design.norm_offset).contiguous()
            return post, L.f32(f"norm{k}", (width,)) if design.pre_norm else None
        self.mixer = M.MIXERS[spec.type](spec.mixer, M.Loader(tensors, prefix + "mix.", dtype, device), width)
        self.post1, self.pre1 = norms(1)
        self.mlp = self.post2 = self.pre2 = None
        if spec.mlp is not None:
            self.mlp = M.MLPS[design.dense_mlp](spec.mlp, M.Loader(tensors, prefix + "mlp.", dtype, device), width)
            self.post2, self.pre2 = norms(2)


@dataclass
class _Between:
    """What happens to the stream ahead of a sublayer."""
    add_embed: bool = False
    add_vec: torch.Tensor | None = None
    norm: torch.Tensor | None = None


class HybridModel:
    DESIGN = HybridDesign()
    DTYPES = (torch.bfloat16, torch.float32)

    def __init__(self, cfg: HybridConfig, tensors, dtype: torch.dtype = torch.bfloat16, device="cuda"):
        """tensors: mapping of stored name -> CPU tensor (safetensors_io.SafeTensors or a dict)."""
        if dtype not in self.DTYPES:
            raise ValueError(f"{dtype} is not supported")
        self.cfg, self.dtype, self.device = cfg, dtype, torch.device(device)
        d = self.DESIGN
        top = M.Loader(tensors, "", dtype, self.device)
        self.embed = top.mat("embed", (cfg.vocab, cfg.width))
        self.head = self.embed if d.tied_head else top.mat("head", (cfg.vocab, cfg.width))
        self.embed_norm = top.f32("embed.norm", (cfg.width,)) if d.embed_norm else None
        self.final_norm = top.f32("final.norm", (cfg.width,))
        self.loop_step = top.f32("loop.step", (cfg.loop.times, cfg.width)) if cfg.loop else None
        self.layers = [_Layer(s, d, tensors, f"l{i}.", cfg.width, dtype, self.device) for i, s in enumerate(cfg.layers)]
        self.runs = cfg.runs()
        self.keep_embed = cfg.loop is not None and cfg.loop.times > 1
        # the sublayers in the order they run: (call, index of its state or None, weights of its output's norm, ends a layer)
        self.steps, self.before = [], []
        for r, (i, t) in enumerate(self.runs):
            l = self.layers[i]
            self.before.append(_Between(t is not None and t > 0, None if t is None else self.loop_step[t].contiguous(), l.pre1))
            self.steps.append((l.mixer, r, l.post1, l.mlp is None))
            if l.mlp is not None:
                self.before.append(_Between(norm=l.pre2))
                self.steps.append((l.mlp, None, l.post2, True))
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
        out = [self.head]
        for fn, _, _, _ in self.steps:
            out += fn.decode_weights() if hasattr(fn, "decode_weights") else [t for t in vars(fn).values() if isinstance(t, torch.Tensor) and t.dim() == 2 and t.dtype == self.dtype]
        return sum(t.numel() * t.element_size() for t in out)

    def new_cache(self, B: int, T_max: int) -> SequenceState:
        return SequenceState([self.layers[i].mixer.state_spec() for i, _ in self.runs], B, T_max, self.dtype, self.device)

    # ---- one step ------------------------------------------------------------------------------------------------
    def hidden(self, ids: torch.Tensor, cache: SequenceState, host_pos: int, layers_out=None) -> torch.Tensor:
        """Residual stream fp32 [B * n, width] after all layers for ids int64 [B, n]; advances cache.pos on the device only."""
        c, off = self.cfg, self.DESIGN.norm_offset
        B, n = ids.shape
        ctx = M.StepContext(B, n, cache.pos, host_pos, c.eps)
        x, h, e = S.embed(self.embed, ids, c.embed_scale, self.embed_norm, off, c.eps, self.keep_embed)
        out = torch.empty(x.shape, dtype=self.dtype, device=self.device) if self.DESIGN.pre_norm or h is not x else None

        def update(y, post, nxt: _Between | None):
            """The stream after y and ahead of the sublayer `nxt`; returns that sublayer's operand."""
            nxt = nxt or _Between()
            S.stream_update(x, self.dtype, c.eps, y, post, c.residual_mult, off, e if nxt.add_embed else None, nxt.add_vec, nxt.norm, out)
            return x if out is None else out
        if self.before and (self.before[0].norm is not None or self.before[0].add_vec is not None):
            h = update(None, None, self.before[0])
        for k, (fn, state, post, ends) in enumerate(self.steps):
            y = fn.forward(h) if state is None else fn.forward(h, cache.layers[state], ctx)
            nxt = self.before[k + 1] if k + 1 < len(self.steps) else None
            if ends and layers_out is not None:
                h = update(y, post, None)
                layers_out.append(x.clone())
                if nxt is not None:
                    h = update(None, None, nxt)
            else:
                h = update(y, post, nxt)
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


class Latodra(HybridModel):
    """Latent attention layers with and without positions, gated GELU feed-forwards, norms on both sides of every sublayer, layer scales, a
    normed and tied embedding, a loop over some of the layers."""
    DESIGN = HybridDesign(dense_mlp="gated_gelu", pre_norm=True, layer_scale=True, embed_norm=True, tied_head=True)


ARCHITECTURES = {c.__name__: c for c in (Gopunex, Latodra)}
