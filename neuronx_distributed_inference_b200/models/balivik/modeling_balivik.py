"""Balivik: a decoder over several residual streams with three kinds of mixers, experts chosen by token id and a repeated span of layers.

``config.json`` lists the layers one by one (``layers[i] = {type, mixer, mlp}``).  A block is :class:`HyperConnectionDecoderLayer`: each
sublayer reads a weighted sum of the ``streams`` copies of the residual stream (RMS norm with one number as weight; the mixer's read also
passes a short causal convolution over time) and its result is written back to all of them while they are mixed.  Parts:

* mixer ``attention`` — :class:`DifferentialAttention`: two softmax maps per head over shared values, subtracted, normalised per head;
* mixer ``lightning`` — :class:`RaggedDecayMixer`: linear attention with a fixed decay per head;
* mixer ``channel_delta`` — :class:`RaggedChannelDeltaMixer`: gated delta rule with a decay per head and key channel from a low-rank
  projection (the ranks are those of the checkpoint's tensors);
* feed-forward ``dense`` — :class:`GatedMLP` (SiLU); ``moe`` — :class:`MoE` with a :class:`TableRouter` and clamped gate-product experts;
* ``loop`` — layers ``start .. stop-1`` run ``times`` times in a row with the same weights, every run with caches and states of its own;
* output: sum of the streams, norm, head, ``logit_scale``.

Every size and constant comes from the checkpoint.  The engine side is the one the other hybrid stacks use: the paged cache with per-run
shapes (:class:`LayeredBlockKVCacheManager`), state lines for everything carried per sequence, ragged rows (prompt portions beside single
decoded tokens) in one forward, decode steps replayed from CUDA graphs.
"""
from __future__ import annotations

import json
import os
from typing import List

import torch
import torch.nn as nn

from ...config import InferenceConfig, NeuronConfig
from ...modules.attention.differential_attention import DifferentialAttention, differential_lambda
from ...modules.checkpoint import tensor_shapes
from ...modules.kvcache import LayeredBlockKVCacheManager
from ...modules.mlp import GatedMLP
from ...modules.moe import ExpertMLPs, MoE, TableRouter
from ...modules.norm import RMSNorm
from ...modules.sampling import Sampler
from ...modules.ssm import RaggedChannelDeltaMixer, RaggedDecayMixer
from ...parallel.layers import ColumnParallelLinear, ParallelEmbedding
from ..application_base import NeuronBaseForCausalLM
from ..model_base import HyperConnectionDecoderLayer, NeuronBaseModel
from ..sodudra.modeling_sodudra import layer_runs

GLU_ALPHA = 1.702        # slope of the sigmoid in the experts' gate product (fixed by the design)
MIXER_TYPES = ("attention", "lightning", "channel_delta")


class BalivikInferenceConfig(InferenceConfig):
    def get_required_attributes(self) -> List[str]:
        return ["layers", "norm", "vocab", "width"]

    def add_derived_config(self):
        self.num_cores_per_group = 1
        self.hidden_size, self.vocab_size, self.num_hidden_layers = self.width, self.vocab, len(self.layers)
        self.rms_norm_eps = float(self.norm["eps"])
        for name, default in (("loop", None), ("canon", None), ("streams", 1), ("logit_scale", 1.0)):
            if not hasattr(self, name):
                setattr(self, name, default)
        self.canon_taps = int((self.canon or {}).get("taps") or 0)
        for i, layer in enumerate(self.layers):
            if layer["type"] not in MIXER_TYPES:
                raise ValueError(f"layer {i}: unknown mixer type {layer['type']!r}")
            mlp = layer.get("mlp")
            if mlp is not None and mlp.get("kind") not in ("dense", "moe"):
                raise ValueError(f"layer {i}: unknown mlp kind {mlp.get('kind')!r}")
        self.runs = layer_runs(len(self.layers), self.loop)

    @classmethod
    def get_neuron_config_cls(cls):
        return NeuronConfig

    @classmethod
    def from_pretrained(cls, model_path: str, neuron_config: NeuronConfig) -> "BalivikInferenceConfig":
        with open(os.path.join(model_path, "config.json")) as f:
            d = json.load(f)
        shapes = tensor_shapes(model_path)
        for i, layer in enumerate(d["layers"]):
            if layer["type"] == "channel_delta":           # the ranks stand in the tensors' shapes only
                for name, tensor in (("decay_rank", "a1"), ("gate_rank", "g1")):
                    if f"l{i}.mix.{tensor}" in shapes:
                        layer["mixer"][name] = shapes[f"l{i}.mix.{tensor}"][0]

        def load(self):
            for k, v in d.items():
                setattr(self, k, v)
        return cls(neuron_config, load_config=load)


class NeuronBalivikModel(NeuronBaseModel):
    meta_extra_keys = ("computed_context_lens",)
    graph_tensor_kwargs = ("slot_mapping", "block_table", "computed_context_lens", "gather_positions")

    def __init__(self, config, device=None):
        super().__init__(config, device)
        # every op of a step is a sync-free kernel launch or a torch op on static shapes (the routed experts run on a device-side
        # permutation with a static row bound); rows with seq_id -1 have q_len 0 and touch neither cache nor state
        self.graph_safe = device is not None and torch.device(device).type == "cuda"

    def setup_attr_for_model(self, config):
        nc = config.neuron_config
        if nc.tp_degree != 1:
            raise NotImplementedError("Balivik: tensor parallel degree 1")
        if not nc.is_block_kv_layout:
            raise ValueError("Balivik runs on the paged KV cache: set is_block_kv_layout=True, pa_block_size, pa_num_blocks")
        self.tp_degree, self.hidden_size = 1, config.width
        self.max_batch_size, self.buckets = nc.max_batch_size, nc.buckets

    def _mixer(self, i, spec, W, eps, dt, dev):
        m = spec["mixer"]
        kw = dict(eps=eps, layer_idx=i, dtype=dt, device=dev, tp_group=self.tp_group)
        heads, dim = m["heads"], m["dim"]
        vdim, kv = m.get("vdim", dim), m.get("kv_heads", heads)
        if spec["type"] == "attention":
            rot = m.get("rot") or {}
            return DifferentialAttention(W, heads, kv, dim, vdim, rot_dims=int(rot.get("dims") or 0), rot_base=float(rot.get("base") or 1.0),
                                         scale=float(m["scale"]) if m.get("scale") is not None else dim ** -0.5,
                                         out_scale=1.0 - float(m["diff"]), **kw)
        if spec["type"] == "lightning":
            return RaggedDecayMixer(W, heads, dim, vdim, m["decay"], **kw)
        return RaggedChannelDeltaMixer(W, heads, kv, dim, vdim, int(m["decay_rank"]), int(m["gate_rank"]), int(m.get("conv") or 1), **kw)

    def _mlp(self, f, config, dt, dev):
        if f is None:
            return None
        W = config.width
        if f["kind"] == "dense":
            return GatedMLP(W, f["ff"], "silu", dt, False, self.tp_group, dev)
        r, e = f["router"], f["expert"]
        experts = ExpertMLPs(r["experts"], W, e["ff"], "clamped_glu", dt, False, dev, act_params=(float(e["limit"]), GLU_ALPHA))
        return MoE(TableRouter(r["experts"], r["top"], config.vocab, dev), experts)

    def init_model(self, config):
        nc = config.neuron_config
        dev, dt = self.device_, nc.torch_dtype
        W, eps = config.width, config.rms_norm_eps
        self.embed_tokens = ParallelEmbedding(config.vocab, W, None, dtype=dt, device=dev, shard_across_embedding=True, pad=True,
                                              tensor_model_parallel_group=self.tp_group)
        norm = lambda: RMSNorm(1, eps, torch.float32, device=dev)       # noqa: E731  (one number for all coordinates)
        layers = []
        for i, spec in enumerate(config.layers):
            mlp = self._mlp(spec.get("mlp"), config, dt, dev)
            layers.append(HyperConnectionDecoderLayer(self._mixer(i, spec, W, eps, dt, dev), mlp, norm(), norm() if mlp is not None else None, W,
                                                      int(config.streams), config.canon_taps, i, dev))
        self.layers = nn.ModuleList(layers)
        self.runs = list(config.runs)
        self.norm = norm()
        self.register_buffer("sum_streams", torch.ones(int(config.streams), dtype=torch.float32, device=dev), persistent=False)
        self.lm_head = ColumnParallelLinear(W, config.vocab, bias=False, gather_output=False, dtype=dt, device=dev, pad=True,
                                            tensor_model_parallel_group=self.tp_group)

    def _kernels_cover_decode(self) -> bool:
        return False

    def init_inference_optimization(self, config):
        nc = self.neuron_config
        if self.on_device_sampling:
            self.sampler = Sampler(nc, self.tp_group, vocab_shard=False)
        # caches and state lines per layer RUN: a layer of the repeated span sees different streams in different passes
        shapes, specs = {}, {}
        for r, (i, _) in enumerate(self.runs):
            kv_shape = getattr(self.layers[i].mixer, "kv_shape", None)
            if kv_shape is not None:
                shapes[r] = kv_shape()
            specs.update(self.layers[i].state_specs(r))
        self.kv_mgr = LayeredBlockKVCacheManager(shapes, {}, nc.pa_num_blocks, nc.pa_block_size, nc.torch_dtype, self.device_,
                                                 state_specs=specs, num_slots=nc.kv_cache_batch_size, state_dtype=nc.torch_dtype)

    # ---- forward hooks ---------------------------------------------------------------------------------------------------
    def build_meta(self, input_ids, attention_mask, position_ids, seq_ids, is_prefill, **kw):
        meta = super().build_meta(input_ids, attention_mask, position_ids, seq_ids, is_prefill, **kw)
        if meta.block_table is None:
            raise ValueError("Balivik: every forward needs block_table (paged KV cache)")
        B, T = input_ids.shape[:2]
        dev = input_ids.device
        q_len = meta.key_valid.sum(-1).to(torch.int32) if meta.key_valid is not None else torch.full((B,), T, dtype=torch.int32, device=dev)
        q_len = torch.where(meta.seq_ids < 0, torch.zeros_like(q_len), q_len)
        ctx = meta.extras.get("computed_context_lens")
        ctx = meta.position_ids[:, 0] if ctx is None else ctx.to(dev)
        meta.extras.update(q_len=q_len.contiguous(), ctx_len=ctx.to(torch.int32).contiguous(), token_ids=input_ids,
                           state_lines=self.kv_mgr.lines_for(meta.seq_ids).to(torch.int32).contiguous(),
                           act_dtype=self.neuron_config.torch_dtype)
        return meta

    def embed(self, input_ids, inputs_embeds=None, vision_embeddings=None, vision_mask=None):
        return super().embed(input_ids, inputs_embeds, vision_embeddings, vision_mask).float()      # fp32 residual streams

    def run_layers(self, x, meta):
        finish = HyperConnectionDecoderLayer.finish
        pending = None
        for r, (i, _) in enumerate(self.runs):
            x, pending = self.layers[i](x, pending, meta, self.kv_mgr, r)
            if meta.capture is not None:
                meta.capture[f"runs.{r}.out"] = finish(x, pending, self.sum_streams)[1]
        return finish(x, pending, self.sum_streams)[1]          # the last sublayer's result joins the streams, which are then summed

    def _finish(self, h, lp_dtype=None):
        return HyperConnectionDecoderLayer.finish(h.float(), None, self.sum_streams[:1], self.norm.weight, self.norm.variance_epsilon, lp_dtype)[1]

    def final_hidden(self, h):
        return self._finish(h)

    def compute_logits(self, h):
        return self.lm_head(self._finish(h, self.neuron_config.torch_dtype)).float() * float(self.config.logit_scale)


class NeuronBalivikForCausalLM(NeuronBaseForCausalLM):
    _model_cls = NeuronBalivikModel
    _STATE_DICT_MODEL_PREFIX = ""

    @classmethod
    def get_config_cls(cls):
        return BalivikInferenceConfig

    @classmethod
    def from_pretrained(cls, model_path: str, neuron_config: NeuronConfig):
        return cls(model_path, BalivikInferenceConfig.from_pretrained(model_path, neuron_config))

    @staticmethod
    def convert_hf_to_neuron_state_dict(sd: dict, config) -> dict:
        """Checkpoint names (``l<i>.mix.q`` ...) -> module parameters: the projections that read the same input stacked for one GEMM, the
        second low-rank projections as one block-diagonal matrix, the experts' matrices stacked along a leading expert axis, the four
        vectors behind a differential attention's lambda folded into that number."""
        one = lambda t: t.reshape(1)          # noqa: E731
        out = {"embed_tokens.weight": sd["embed"], "lm_head.weight": sd["head"], "norm.weight": one(sd["final.norm"])}
        for i, spec in enumerate(config.layers):
            a, b = f"l{i}.", f"layers.{i}."
            f = spec.get("mlp")
            for q in (1, 2) if f is not None else (1,):
                out[f"{b}norm{q}.weight"] = one(sd[f"{a}norm{q}"])
                for n in ("in", "out", "mix"):
                    out[f"{b}{n}{q}"] = sd[f"{a}hc{q}.{n}"]
            if config.canon_taps:
                out[b + "conv1_weight"] = sd[a + "canon1"]
            x, y, m = a + "mix.", b + "mixer.", spec["mixer"]
            cat = lambda *names: torch.cat([sd[x + n] for n in names], 0)          # noqa: E731
            if spec["type"] == "attention":
                out[y + "in_proj.weight"] = cat("q", "k", "v")
                out[y + "o_proj.weight"] = sd[x + "o"]
                out[y + "lam"] = differential_lambda(sd[x + "lq1"], sd[x + "lk1"], sd[x + "lq2"], sd[x + "lk2"], float(m["diff"]))
            elif spec["type"] == "lightning":
                out[y + "in_proj.weight"] = cat("q", "k", "v", "g")
                out[y + "norm_weight"], out[y + "out_proj.weight"] = sd[x + "norm"], sd[x + "o"]
            else:
                out[y + "in_proj.weight"] = cat("q", "k", "v", "b", "a1", "g1")
                out[y + "low_rank_up.weight"] = RaggedChannelDeltaMixer.block_diagonal(sd[x + "a2"], sd[x + "g2"])
                ident = lambda n: torch.ones(sd[x + n].shape[0], 1, dtype=sd[x + n].dtype)          # noqa: E731  (no convolution: one tap of one)
                out[y + "conv_weight"] = torch.cat([sd[x + n + ".conv"] if x + n + ".conv" in sd else ident(n) for n in ("q", "k", "v")], 0)
                for src, dst in (("A_log", "A_log"), ("dt_bias", "dt_bias"), ("norm", "norm_weight"), ("o", "out_proj.weight")):
                    out[y + dst] = sd[x + src]
            if f is None:
                continue
            x, y = a + "mlp.", b + "mlp."
            if f["kind"] == "dense":
                out[y + "gate_up_proj.weight"] = torch.cat([sd[x + "gate"], sd[x + "up"]], 0)
                out[y + "down_proj.weight"] = sd[x + "down"]
            else:
                E = f["router"]["experts"]
                out[y + "router.table"] = sd[x + "table"].to(torch.int32)
                out[y + "expert_mlps.gate_up_proj"] = torch.stack([torch.cat([sd[f"{x}e{e}.gate"], sd[f"{x}e{e}.up"]], 0) for e in range(E)], 0)
                out[y + "expert_mlps.down_proj"] = torch.stack([sd[f"{x}e{e}.down"] for e in range(E)], 0)
        return out

    def init_random_weights(self, seed: int = 0):
        """Benchmarks: N(0, 0.02) projections, unit norms, streams that are averaged and copied, small convolution taps, experts dealt out in turn."""
        super().init_random_weights(seed)
        S = int(self.config.streams)
        with torch.no_grad():
            for name, p in self.model.named_parameters():
                leaf = name.rsplit(".", 1)[-1]
                if name.endswith(("norm1.weight", "norm2.weight", "norm_weight")) or name == "norm.weight" or leaf in ("out1", "out2"):
                    p.fill_(1.0)
                elif leaf in ("in1", "in2"):
                    p.fill_(1.0 / S)
                elif leaf in ("mix1", "mix2"):
                    p.copy_(torch.eye(S))
                elif leaf == "conv1_weight":
                    p.fill_(0.1)
                elif leaf == "conv_weight":
                    p.fill_(1.0 / p.shape[1])
                elif leaf == "A_log":
                    p.zero_()
                elif leaf == "dt_bias":
                    p.fill_(-2.0)
                elif leaf == "lam":
                    p.fill_(0.3)
                elif leaf == "table":
                    i = int(name.split(".")[1])
                    E, k = self.config.layers[i]["mlp"]["router"]["experts"], p.shape[1]
                    rows = torch.arange(p.shape[0]).view(-1, 1) * k + torch.arange(k).view(1, k) + 7 * i
                    p.copy_((rows % E).to(torch.int32))
