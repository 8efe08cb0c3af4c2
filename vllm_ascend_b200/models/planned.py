"""Decoder built from a layer plan (``ModelConfig.layer_plan``): every layer has its own mixer and sizes.

What the plan's layers have in common:

* the residual stream is fp32; a norm stands in front of every sub-layer (``pre_norm``) and, with
  ``sandwich_norm``, behind it, ``r += m post(f(pre(r)))`` with m = ``residual_multiplier``, and one kernel does
  the token-wise work between two sub-layers (``ops.stream.stream_norm``);
* with ``residual_streams`` there are several parallel streams per token, mixed by learned weights at every
  sub-layer (``ops.stream.stream_mix``);
* mixers are the framework's: latent attention (``MLAAttention`` with window and sink, or over another layer's
  latents), the gated delta rule (``GatedDeltaNet``), paged attention with options (``VariantAttention``), HGRN2
  (``HGRN2Mixer``) and attention beside a Mamba-2 state space (``ParallelMixer``); so
  are the feed-forwards (gated, plain, mixture of experts); each is built from ``ModelConfig.layer_config(i)``;
* optional learned positions (``learned_positions``): a vector per position added to the embeddings;
* optional per-layer token input (``token_side_dim``): a slice of a second embedding table, gated by the
  stream, projected, RMS-normed and added after the layer's sub-layers;
* optional loop (``layer_loop``): some layers run several times with the same weights; with
  ``layer_loop_refeed`` the embedding output is added to the stream again before each pass but the first;
* layers that use another layer's parameters (``weights_of`` of a plan's entry).

``layers`` lists the layer *runs* in execution order: a looped layer appears once per pass, and the layer whose
parameters others use once for each of them, so every run has its own entry in the runner's cache list while the
parameters are shared.
"""
from __future__ import annotations

from typing import Iterable, Optional

import torch

from ..config import ModelConfig
from ..layer_plan import run_order
from ..ops.stream import PLAIN, NormSpec, StreamMix, side_gate, stream_mix, stream_norm
from ..parallel import state as pstate
from .gdn import GatedDeltaNet
from .hgrn2 import HGRN2Mixer
from .layers import (Linear, ParallelLMHead, ParamFactory, PlainMLP, SwiGLUMLP, TPComm, VocabParallelEmbedding,
                     copy_exact)
from .parallel_mixer import ParallelMixer
from .transformer import MLAAttention, SparseMoeBlock
from .variant_attention import VariantAttention

#: mixer kind of a plan -> constructor (param factory, layer config, layer index, comm, max positions)
MIXERS = {
    "latent": lambda pf, cfg, i, comm, max_pos: MLAAttention(pf, cfg, i, comm, max_pos),
    "delta": lambda pf, cfg, i, comm, max_pos: GatedDeltaNet(pf, cfg, i, comm),
    "attention": lambda pf, cfg, i, comm, max_pos: VariantAttention(pf, cfg, i, comm, max_pos),
    "parallel": lambda pf, cfg, i, comm, max_pos: ParallelMixer(pf, cfg, i, comm, max_pos),
    "hgrn2": lambda pf, cfg, i, comm, max_pos: HGRN2Mixer(pf, cfg, i, comm),
}


#: checkpoint name -> attribute of a sub-layer's stream mixing weights
_MIX_PARTS = {"in": "read", "out": "write", "mix": "mix"}


def _norm(pf: ParamFactory, cfg: ModelConfig, kind: Optional[str] = None) -> NormSpec:
    kind = kind or cfg.norm_type
    bias = kind == "layer" and cfg.norm_bias
    return NormSpec(kind, pf.ones((cfg.hidden_size,)), pf.zeros((cfg.hidden_size,)) if bias else None,
                    cfg.norm_groups if kind == "rms" else 1)


def _feed_forward(pf: ParamFactory, lcfg: ModelConfig, idx: int, comm: TPComm, ep_group, moe_runtime):
    prefix = f"model.layers.{idx}.mlp"
    if lcfg.is_moe:
        ranks = 1 if ep_group is not None and ep_group.world_size > 1 else comm.size
        if lcfg.moe_intermediate_size % ranks or lcfg.shared_expert_intermediate_size % comm.size:
            raise ValueError(f"layer {idx}: experts do not divide over {comm.size} tensor-parallel ranks")
        return SparseMoeBlock(pf, lcfg, idx, comm, ep_group, moe_runtime)
    kind = SwiGLUMLP if lcfg.mlp_gated else PlainMLP
    return kind(pf, prefix, lcfg.hidden_size, lcfg.intermediate_size, comm, act=lcfg.hidden_act)


class TokenSide:
    """Per-layer token input: y = proj (gelu_tanh(gate r) * slice of the token's row), joined through an RMS
    norm.  Replicated over TP."""

    def __init__(self, pf: ParamFactory, cfg: ModelConfig, layer_idx: int, table: torch.Tensor):
        p, D = f"model.layers.{layer_idx}.side", cfg.token_side_dim
        self.table, self.offset = table, layer_idx * D
        self.gate = Linear(pf.normal(f"{p}.gate", (D, cfg.hidden_size)), name=f"{p}.gate")
        self.proj = Linear(pf.normal(f"{p}.proj", (cfg.hidden_size, D)), name=f"{p}.proj")
        self.norm = _norm(pf, cfg, "rms")

    def __call__(self, x: torch.Tensor, ids: torch.Tensor) -> torch.Tensor:
        return self.proj(side_gate(self.gate(x), ids, self.table, self.offset))


def _stream_mix(pf: ParamFactory, prefix: str, streams: int) -> StreamMix:
    """Mixing weights of a sub-layer.  Random models start near one stream per residual sum."""
    f32 = torch.float32
    mix = torch.eye(streams, dtype=f32, device=pf.device)
    if streams > 1:
        mix = 0.9 * mix + pf.normal(f"{prefix}.mix", (streams, streams), std=0.05, dtype=f32)
    return StreamMix(pf.ones((streams,), f32) / streams, pf.ones((streams,), f32), mix.contiguous())


class PlannedLayer:
    def __init__(self, pf: ParamFactory, cfg: ModelConfig, idx: int, comm: TPComm, max_pos: int,
                 side_table: Optional[torch.Tensor], ep_group=None, moe_runtime=None):
        entry, lcfg = cfg.layer_plan[idx], cfg.layer_config(idx)
        linear = entry["mixer"] in ("delta", "hgrn2")
        heads = lcfg.linear_num_key_heads if linear else lcfg.num_attention_heads
        if heads % comm.size or (linear and lcfg.linear_num_value_heads % comm.size):
            raise ValueError(f"layer {idx}: heads do not divide over {comm.size} tensor-parallel ranks")
        self.idx = idx
        self.self_attn = MIXERS[entry["mixer"]](pf, lcfg, idx, comm, max_pos)
        streams = cfg.residual_streams
        # in front of and behind a sub-layer
        self.norm1, self.norm1b = (_norm(pf, cfg) if on else PLAIN for on in (cfg.pre_norm, cfg.sandwich_norm))
        self.hc1 = _stream_mix(pf, f"model.layers.{idx}.hc1", streams) if streams else None
        self.mlp = self.norm2 = self.norm2b = self.hc2 = None
        if entry["mlp"]:
            self.norm2, self.norm2b = (_norm(pf, cfg) if on else PLAIN for on in (cfg.pre_norm, cfg.sandwich_norm))
            self.hc2 = _stream_mix(pf, f"model.layers.{idx}.hc2", streams) if streams else None
            self.mlp = _feed_forward(pf, lcfg, idx, comm, ep_group, moe_runtime)
        self.side = TokenSide(pf, cfg, idx, side_table) if side_table is not None else None

    def norms(self) -> dict[str, NormSpec]:
        """The layer's norms under their checkpoint names: a sub-layer's only norm has no suffix."""
        out = {}
        for k, pre, post in ((1, self.norm1, self.norm1b), (2, self.norm2, self.norm2b)):
            here = [n for n in (pre, post) if n is not None and n is not PLAIN]
            out.update(zip((f"norm{k}", f"norm{k}b"), here))
        return out

    def mixes(self) -> dict[str, StreamMix]:
        return {k: m for k, m in (("hc1", self.hc1), ("hc2", self.hc2)) if m is not None}


class PlannedCausalLM:
    """Model object the runner drives: ``forward`` -> hidden states, ``compute_logits``."""

    def __init__(self, cfg: ModelConfig, device, max_model_len: int = 4096,
                 tp_group: Optional[pstate.GroupCoordinator] = None, ep_group=None, moe_runtime=None,
                 layer_range: Optional[tuple[int, int]] = None):
        if layer_range is not None and layer_range != (0, cfg.num_hidden_layers):
            raise NotImplementedError("decoders built from a layer plan are not split into pipeline stages")
        if cfg.quantization:
            raise NotImplementedError("decoders built from a layer plan are served unquantized")
        from ..parallel import finegrained as fgm
        from ..platform_config import get_b200_config
        if fgm.get_fg() is not None or get_b200_config().weight_offload_config.enabled:
            raise NotImplementedError("decoders built from a layer plan take neither fine-grained tensor "
                                      "parallelism nor weight offloading")
        self.cfg = cfg
        self.device = torch.device(device)
        self.dtype = cfg.torch_dtype
        if self.dtype not in (torch.bfloat16, torch.float32):
            raise ValueError(f"activations are bfloat16 or float32, not {cfg.dtype}")
        pf = ParamFactory(cfg, self.device, self.dtype)
        self.comm = TPComm(tp_group or pstate.get_tp_group())
        self.sp_ctx = None
        self.layer_hook = None             # callable(layer run index), run after each layer run
        self.aux_layers = self.aux_hidden = None
        self.is_first = self.is_last = True
        self.layer_range = (0, cfg.num_hidden_layers)
        self.embed_tokens = VocabParallelEmbedding(pf, "model.embed_tokens", cfg.vocab_size, cfg.hidden_size, self.comm)
        self.side_embed = None
        if cfg.token_side_dim:
            self.side_embed = pf.normal("model.side_embed", (cfg.vocab_size, cfg.num_hidden_layers * cfg.token_side_dim))
        self.pos_embed = None
        if cfg.learned_positions:
            self.pos_embed = pf.normal("model.pos_embed", (cfg.learned_positions, cfg.hidden_size))
        max_pos = max(max_model_len, 16)
        if moe_runtime is not None:
            sizes = {(c.num_experts, c.num_experts_per_tok, c.moe_intermediate_size)
                     for c in map(cfg.layer_config, range(cfg.num_hidden_layers)) if c.is_moe}
            if len(sizes) > 1:
                raise NotImplementedError("expert parallelism takes layers whose experts are alike")
        owner = [entry.get("weights_of", i) for i, entry in enumerate(cfg.layer_plan)]
        own = {i: PlannedLayer(pf, cfg, i, self.comm, max_pos, self.side_embed, ep_group, moe_runtime)
               for i in sorted(set(owner))}
        self.unique_layers = list(own.values())
        order, again = run_order(cfg.num_hidden_layers, cfg.layer_loop)
        self.fed_again = again if cfg.layer_loop_refeed else set()
        self.layers = [own[owner[i]] for i in order]
        self._layer_of = own
        self.norm = _norm(pf, cfg)
        if cfg.residual_streams and (cfg.token_side_dim or self.fed_again):
            raise NotImplementedError("parallel streams take neither a token side input nor a second embedding feed")
        if cfg.residual_streams and cfg.residual_multiplier != 1.0:
            raise NotImplementedError("parallel streams have write weights instead of a residual multiplier")
        if cfg.learned_positions and not cfg.residual_streams:
            raise NotImplementedError("learned positions join the embeddings of decoders with residual streams")
        self.lm_head = ParallelLMHead(self.embed_tokens if cfg.tie_word_embeddings else VocabParallelEmbedding(
            pf, "lm_head", cfg.vocab_size, cfg.hidden_size, self.comm))

    # -- forward ---------------------------------------------------------
    def forward(self, input_ids: torch.Tensor, meta, kv_caches: list, intermediate=None,
                inputs_embeds: Optional[torch.Tensor] = None):
        cfg, eps, dtype = self.cfg, self.cfg.rms_norm_eps, self.dtype
        T = input_ids.shape[0]
        # the embedding output: gathered from the table inside the stream kernel where the table is whole
        if inputs_embeds is not None:
            emb = dict(embed=inputs_embeds.to(dtype))
        elif self.comm.size > 1:
            emb = dict(embed=self.embed_tokens(input_ids), embed_scale=cfg.embed_scale)
        else:
            emb = dict(embed=self.embed_tokens.weight[:cfg.vocab_size], ids=input_ids, embed_scale=cfg.embed_scale)
        if cfg.residual_streams:
            return self._forward_streams(T, emb, None if inputs_embeds is not None else self.pos_embed, meta, kv_caches)
        r = torch.empty((T, cfg.hidden_size), dtype=torch.float32, device=input_ids.device)
        x = stream_norm(r, None, None, self.layers[0].norm1, eps, dtype, embed_set=True, **emb)
        last, m = len(self.layers) - 1, cfg.residual_multiplier
        self.stream = r if self.layer_hook is not None else None
        for run, (layer, cache) in enumerate(zip(self.layers, kv_caches)):
            y, post = layer.self_attn(x, meta, cache), layer.norm1b
            if layer.mlp is not None:
                x = stream_norm(r, y, post, layer.norm2, eps, dtype, post_scale=m)
                y, post = layer.mlp(x), layer.norm2b
            if layer.side is not None:
                x = stream_norm(r, y, post, PLAIN, eps, dtype, post_scale=m)
                y, post = layer.side(x, input_ids), layer.side.norm
            nxt = self.layers[run + 1].norm1 if run < last else self.norm
            if self.layer_hook is not None:      # the hook sees the stream before the next pass is fed again
                stream_norm(r, y, post, None, eps, dtype, post_scale=m)
                self.layer_hook(run)
                y = post = None
            x = stream_norm(r, y, post, nxt, eps, dtype, post_scale=m, **(emb if run + 1 in self.fed_again else {}))
        return x

    def _forward_streams(self, T: int, emb: dict, pos_table: Optional[torch.Tensor], meta, kv_caches: list):
        """Layers on ``residual_streams`` parallel streams: a sub-layer reads a weighted sum of them, and its output
        and the old streams make the new ones."""
        eps, dtype, layers = self.cfg.rms_norm_eps, self.dtype, self.layers
        r = torch.empty((T, self.cfg.residual_streams, self.cfg.hidden_size), dtype=torch.float32, device=self.device)
        x = stream_mix(r, None, None, None, layers[0].hc1, layers[0].norm1, eps, dtype, pos_table=pos_table,
                       positions=meta.positions[:T], **emb)
        for run, (layer, cache) in enumerate(zip(layers, kv_caches)):
            y, post, joined = layer.self_attn(x, meta, cache), layer.norm1b, layer.hc1
            if layer.mlp is not None:
                x = stream_mix(r, y, post, joined, layer.hc2, layer.norm2, eps, dtype)
                y, post, joined = layer.mlp(x), layer.norm2b, layer.hc2
            nxt = layers[run + 1] if run + 1 < len(layers) else None
            if self.layer_hook is not None:
                stream_mix(r, y, post, joined, None, None, eps, dtype)
                self.stream = r.sum(1)
                self.layer_hook(run)
                y = post = joined = None
            x = stream_mix(r, y, post, joined, nxt and nxt.hc1, nxt.norm1 if nxt else self.norm, eps, dtype,
                           store=nxt is not None)
        return x

    __call__ = forward

    def compute_logits(self, hidden: torch.Tensor) -> torch.Tensor:
        return self.lm_head(hidden)

    def embed_input_ids(self, input_ids: torch.Tensor) -> torch.Tensor:
        """Rows of the embedding output, as ``inputs_embeds`` takes them."""
        if self.pos_embed is not None:
            raise NotImplementedError("the embedding output depends on the positions as well")
        return self.embed_tokens(input_ids) * self.cfg.embed_scale

    # -- parameters --------------------------------------------------------
    def named_parameters(self):
        yield "model.embed_tokens.weight", self.embed_tokens.weight
        if self.side_embed is not None:
            yield "model.side_embed.weight", self.side_embed
        if self.pos_embed is not None:
            yield "model.pos_embed.weight", self.pos_embed
        for L in self.unique_layers:
            p, a = f"model.layers.{L.idx}", L.self_attn
            for name, n in L.norms().items():
                yield f"{p}.{name}.weight", n.weight
                if n.bias is not None:
                    yield f"{p}.{name}.bias", n.bias
            for name, m in L.mixes().items():
                for n in m.__slots__:
                    yield f"{p}.{name}.{n}", getattr(m, n)
            whole = (VariantAttention, ParallelMixer, HGRN2Mixer)      # list all of their tensors themselves
            if isinstance(a, whole):
                for n, t in a.named_tensors():
                    yield f"{p}.self_attn.{n}", t
            for attr in () if isinstance(a, whole) else (
                    "in_proj_qkvz", "in_proj_ba", "out_proj", "q_proj", "q_a_proj", "q_b_proj", "kv_a_proj", "kv_b_proj",
                    "o_proj"):
                lin = getattr(a, attr, None)
                if isinstance(lin, Linear):
                    for n, t in lin.named_tensors():
                        yield f"{p}.self_attn.{attr}.{n}", t
            if isinstance(a, GatedDeltaNet):
                for n, t in a.named_tensors():
                    yield f"{p}.self_attn.{n}", t
            elif isinstance(a, MLAAttention):
                for attr in ("q_a_norm", "kv_a_norm"):
                    if getattr(a, attr, None) is not None:
                        yield f"{p}.self_attn.{attr}.weight", getattr(a, attr).weight
                if a.sink is not None:
                    yield f"{p}.self_attn.sink", a.sink
            if L.mlp is not None:
                for n, t in L.mlp.named_tensors():
                    yield f"{p}.mlp.{n}", t
            if L.side is not None:
                yield f"{p}.side.gate.weight", L.side.gate.weight
                yield f"{p}.side.proj.weight", L.side.proj.weight
                yield f"{p}.side.norm.weight", L.side.norm.weight
        yield "model.norm.weight", self.norm.weight
        if self.norm.bias is not None:
            yield "model.norm.bias", self.norm.bias
        if not self.cfg.tie_word_embeddings:
            yield "lm_head.weight", self.lm_head.weight

    def num_parameters(self) -> int:
        return sum(t.numel() for _, t in self.named_parameters())

    # -- checkpoint loading ------------------------------------------------
    def tensor_names(self) -> set[str]:
        """Names of the tensors a checkpoint of this model has."""
        def norm(name, n):
            return {name} | ({name + ".b"} if n.bias is not None else set())
        out = {"embed"} | norm("final.norm", self.norm)
        if not self.cfg.tie_word_embeddings:
            out.add("head")
        if self.pos_embed is not None:
            out.add("pos")
        if self.side_embed is not None:
            out.add("side.embed")
        for L in self.unique_layers:
            p = f"l{L.idx}."
            for name, n in L.norms().items():
                out |= norm(p + name, n)
            out |= {f"{p}{name}.{part}" for name in L.mixes() for part in _MIX_PARTS}
            out |= {p + "mix." + part for part in L.self_attn.parts()}
            if L.mlp is not None:
                out |= {p + "mlp." + part for part in L.mlp.parts()}
            if L.side is not None:
                out |= {p + "side." + part for part in ("gate", "proj", "norm")}
        return out

    def check_loaded(self, loaded: set[str]) -> None:
        missing = sorted(self.tensor_names() - loaded)
        if self.cfg.residual_streams == 1:           # one stream without weights is a plain residual sum
            missing = [n for n in missing if ".hc" not in n]
        if missing:
            raise ValueError(f"checkpoint lacks {len(missing)} tensors: {', '.join(missing[:8])}")

    def load_weights(self, weights: Iterable[tuple[str, torch.Tensor]]) -> set[str]:
        loaded, known = set(), self.tensor_names()
        for name, w in weights:
            if name not in known:
                own = dict(self.named_parameters()).get(name)      # parameters under this package's names
                if own is None:
                    raise ValueError(f"unexpected tensor {name!r}")
                copy_exact(own, w, name)
            else:
                self._load_one(name, w)
            loaded.add(name)
        for L in self.unique_layers:
            if hasattr(L.self_attn, "process_weights_after_loading"):
                L.self_attn.process_weights_after_loading()
        return loaded

    def _load_one(self, name: str, w: torch.Tensor) -> None:
        def norm(n: NormSpec, which: str):
            copy_exact(n.bias if which == "b" else n.weight, w, name)
        if name in ("embed", "head"):
            e = self.embed_tokens if name == "embed" else self.lm_head.embed
            if tuple(w.shape) != (self.cfg.vocab_size, self.cfg.hidden_size):
                raise ValueError(f"tensor {name}: unexpected shape {tuple(w.shape)}")
            rows = w[e.start:e.start + e.shard]
            e.weight[:rows.shape[0]].copy_(rows)
            return None
        if name == "pos":
            return copy_exact(self.pos_embed, w, name)
        if name == "side.embed":
            return copy_exact(self.side_embed, w, name)
        if name.startswith("final.norm"):
            return norm(self.norm, name[len("final.norm."):])
        layer, _, rest = name.partition(".")
        L = self._layer_of[int(layer[1:])]
        group, _, part = rest.partition(".")
        if group == "mix":
            return L.self_attn.load_part(part, w)
        if group in L.mixes():
            return copy_exact(getattr(L.mixes()[group], _MIX_PARTS[part]), w, name)
        if group == "side":
            return norm(L.side.norm, "") if part == "norm" else copy_exact(getattr(L.side, part).weight, w, name)
        if group == "mlp":
            return L.mlp.load_part(part, w)
        return norm(L.norms()[group], part)
