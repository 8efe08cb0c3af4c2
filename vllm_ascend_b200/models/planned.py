"""Decoder built from a layer plan (``ModelConfig.layer_plan``): every layer has its own mixer and sizes.

What the plan's layers have in common:

* the residual stream is fp32; a norm stands in front of and behind every sub-layer,
  ``r += post(f(pre(r)))``, and one kernel does the token-wise work between two sub-layers
  (``ops.stream.stream_norm``);
* mixers are the framework's: latent attention (``MLAAttention`` with window and sink) and the gated delta
  rule (``GatedDeltaNet``), each built from ``ModelConfig.layer_config(i)``;
* optional per-layer token input (``token_side_dim``): a slice of a second embedding table, gated by the
  stream, projected, RMS-normed and added after the layer's sub-layers;
* optional loop (``layer_loop``): some layers run several times with the same weights; before each pass but
  the first the embedding output is added to the stream again.

``layers`` lists the layer *runs* in execution order: a looped layer appears once per pass, so every pass
has its own entry in the runner's cache list while the parameters are shared.
"""
from __future__ import annotations

from typing import Iterable, Optional

import torch

from ..config import ModelConfig
from ..layer_plan import run_order
from ..ops.stream import PLAIN, NormSpec, side_gate, stream_norm
from ..parallel import state as pstate
from .gdn import GatedDeltaNet
from .layers import (Linear, ParallelLMHead, ParamFactory, SwiGLUMLP, TPComm, VocabParallelEmbedding, copy_exact)
from .transformer import MLAAttention

#: mixer kind of a plan -> constructor (param factory, layer config, layer index, comm, max positions)
MIXERS = {
    "latent": lambda pf, cfg, i, comm, max_pos: MLAAttention(pf, cfg, i, comm, max_pos),
    "delta": lambda pf, cfg, i, comm, max_pos: GatedDeltaNet(pf, cfg, i, comm),
}


def _norm(pf: ParamFactory, cfg: ModelConfig, kind: Optional[str] = None) -> NormSpec:
    kind = kind or cfg.norm_type
    return NormSpec(kind, pf.ones((cfg.hidden_size,)), pf.zeros((cfg.hidden_size,)) if kind == "layer" else None)


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


class PlannedLayer:
    def __init__(self, pf: ParamFactory, cfg: ModelConfig, idx: int, comm: TPComm, max_pos: int,
                 side_table: Optional[torch.Tensor]):
        entry, lcfg = cfg.layer_plan[idx], cfg.layer_config(idx)
        heads = lcfg.linear_num_key_heads if entry["mixer"] == "delta" else lcfg.num_attention_heads
        if heads % comm.size or (entry["mixer"] == "delta" and lcfg.linear_num_value_heads % comm.size):
            raise ValueError(f"layer {idx}: heads do not divide over {comm.size} tensor-parallel ranks")
        self.idx = idx
        self.self_attn = MIXERS[entry["mixer"]](pf, lcfg, idx, comm, max_pos)
        self.norm1, self.norm1b = _norm(pf, cfg), _norm(pf, cfg)
        self.mlp = self.norm2 = self.norm2b = None
        if entry["mlp"]:
            self.norm2, self.norm2b = _norm(pf, cfg), _norm(pf, cfg)
            self.mlp = SwiGLUMLP(pf, f"model.layers.{idx}.mlp", cfg.hidden_size, lcfg.intermediate_size, comm,
                                 act=cfg.hidden_act)
        self.side = TokenSide(pf, cfg, idx, side_table) if side_table is not None else None

    def norms(self) -> dict[str, NormSpec]:
        out = {"norm1": self.norm1, "norm1b": self.norm1b}
        if self.mlp is not None:
            out.update(norm2=self.norm2, norm2b=self.norm2b)
        return out


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
        max_pos = max(max_model_len, 16)
        self.unique_layers = [PlannedLayer(pf, cfg, i, self.comm, max_pos, self.side_embed)
                              for i in range(cfg.num_hidden_layers)]
        order, self.fed_again = run_order(cfg.num_hidden_layers, cfg.layer_loop)
        self.layers = [self.unique_layers[i] for i in order]
        self.norm = _norm(pf, cfg)
        head = VocabParallelEmbedding(pf, "lm_head", cfg.vocab_size, cfg.hidden_size, self.comm)
        self.lm_head = ParallelLMHead(head)

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
        r = torch.empty((T, cfg.hidden_size), dtype=torch.float32, device=input_ids.device)
        x = stream_norm(r, None, None, self.layers[0].norm1, eps, dtype, embed_set=True, **emb)
        last = len(self.layers) - 1
        for run, (layer, cache) in enumerate(zip(self.layers, kv_caches)):
            y, post = layer.self_attn(x, meta, cache), layer.norm1b
            if layer.mlp is not None:
                x = stream_norm(r, y, post, layer.norm2, eps, dtype)
                y, post = layer.mlp(x), layer.norm2b
            if layer.side is not None:
                x = stream_norm(r, y, post, PLAIN, eps, dtype)
                y, post = layer.side(x, input_ids), layer.side.norm
            nxt = self.layers[run + 1].norm1 if run < last else self.norm
            if self.layer_hook is not None:      # the hook sees the stream before the next pass is fed again
                stream_norm(r, y, post, None, eps, dtype)
                self.layer_hook(run)
                y = post = None
            x = stream_norm(r, y, post, nxt, eps, dtype, **(emb if run + 1 in self.fed_again else {}))
        self.stream = r if self.layer_hook is not None else None
        return x

    __call__ = forward

    def compute_logits(self, hidden: torch.Tensor) -> torch.Tensor:
        return self.lm_head(hidden)

    def embed_input_ids(self, input_ids: torch.Tensor) -> torch.Tensor:
        """Rows of the embedding output, as ``inputs_embeds`` takes them."""
        return self.embed_tokens(input_ids) * self.cfg.embed_scale

    # -- parameters --------------------------------------------------------
    def named_parameters(self):
        yield "model.embed_tokens.weight", self.embed_tokens.weight
        if self.side_embed is not None:
            yield "model.side_embed.weight", self.side_embed
        for L in self.unique_layers:
            p, a = f"model.layers.{L.idx}", L.self_attn
            for name, n in L.norms().items():
                yield f"{p}.{name}.weight", n.weight
                if n.bias is not None:
                    yield f"{p}.{name}.bias", n.bias
            for attr in ("in_proj_qkvz", "in_proj_ba", "out_proj", "q_proj", "kv_a_proj", "kv_b_proj", "o_proj"):
                lin = getattr(a, attr, None)
                if isinstance(lin, Linear):
                    for n, t in lin.named_tensors():
                        yield f"{p}.self_attn.{attr}.{n}", t
            if getattr(a, "is_linear_attention", False):
                for n, t in a.named_tensors():
                    yield f"{p}.self_attn.{n}", t
            else:
                yield f"{p}.self_attn.kv_a_norm.weight", a.kv_a_norm.weight
                if a.sink is not None:
                    yield f"{p}.self_attn.sink", a.sink
            if L.mlp is not None:
                for attr in ("gate_up_proj", "down_proj"):
                    for n, t in getattr(L.mlp, attr).named_tensors():
                        yield f"{p}.mlp.{attr}.{n}", t
            if L.side is not None:
                yield f"{p}.side.gate.weight", L.side.gate.weight
                yield f"{p}.side.proj.weight", L.side.proj.weight
                yield f"{p}.side.norm.weight", L.side.norm.weight
        yield "model.norm.weight", self.norm.weight
        if self.norm.bias is not None:
            yield "model.norm.bias", self.norm.bias
        yield "lm_head.weight", self.lm_head.weight

    def num_parameters(self) -> int:
        return sum(t.numel() for _, t in self.named_parameters())

    # -- checkpoint loading ------------------------------------------------
    def tensor_names(self) -> set[str]:
        """Names of the tensors a checkpoint of this model has."""
        def norm(name, n):
            return {name} | ({name + ".b"} if n.bias is not None else set())
        out = {"embed", "head"} | norm("final.norm", self.norm)
        if self.side_embed is not None:
            out.add("side.embed")
        for L in self.unique_layers:
            p = f"l{L.idx}."
            for name, n in L.norms().items():
                out |= norm(p + name, n)
            out |= {p + "mix." + part for part in L.self_attn.parts()}
            if L.mlp is not None:
                out |= {p + "mlp." + part for part in ("gate", "up", "down")}
            if L.side is not None:
                out |= {p + "side." + part for part in ("gate", "proj", "norm")}
        return out

    def check_loaded(self, loaded: set[str]) -> None:
        missing = sorted(self.tensor_names() - loaded)
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
            if isinstance(L.self_attn, MLAAttention):
                L.self_attn.process_weights_after_loading()
        return loaded

    def _load_one(self, name: str, w: torch.Tensor) -> None:
        tp, r = self.comm.size, self.comm.rank

        def norm(n: NormSpec, which: str):
            copy_exact(n.bias if which == "b" else n.weight, w, name)
        if name in ("embed", "head"):
            e = self.embed_tokens if name == "embed" else self.lm_head.embed
            if tuple(w.shape) != (self.cfg.vocab_size, self.cfg.hidden_size):
                raise ValueError(f"tensor {name}: unexpected shape {tuple(w.shape)}")
            rows = w[e.start:e.start + e.shard]
            e.weight[:rows.shape[0]].copy_(rows)
            return None
        if name == "side.embed":
            return copy_exact(self.side_embed, w, name)
        if name.startswith("final.norm"):
            return norm(self.norm, name[len("final.norm."):])
        layer, _, rest = name.partition(".")
        L = self.unique_layers[int(layer[1:])]
        group, _, part = rest.partition(".")
        if group == "mix":
            return L.self_attn.load_part(part, w)
        if group == "side":
            return norm(L.side.norm, "") if part == "norm" else copy_exact(getattr(L.side, part).weight, w, name)
        if group == "mlp":
            if part == "down":
                n = w.shape[1] // tp
                return copy_exact(L.mlp.down_proj.weight, w[:, r * n:(r + 1) * n], name)
            n = w.shape[0] // tp
            at = 0 if part == "gate" else n
            return copy_exact(L.mlp.gate_up_proj.weight[at:at + n], w[r * n:(r + 1) * n], name)
        return norm(L.norms()[group], part)
