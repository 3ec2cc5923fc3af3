"""Navulorn: a post-norm decoder with bigram embeddings over window attention, latent attention and matrix memories.

``config.json`` lists the layers one by one (``layers[i] = {type, mixer, mlp}``); a layer is ``x <- norm1(alpha x + mixer(x))`` followed, when
it has a feed-forward, by ``x <- norm2(alpha x + mlp(x))`` (:class:`PostNormDecoderLayer`, fp32 stream, plain norm weights).  Parts:

* embedding — ``embed[token] * scale`` plus, when the configuration has one, row ``(previous * mul_prev + token * mul_cur) mod buckets`` of
  a bigram table (its last row for a sequence's first token); the previous token is carried per sequence in a state line;
* mixer ``attention`` — :class:`ConvWindowAttention` without convolution: q / k RMS norm over whole rows, rotate-half rotation of the first
  ``rot.dims`` channels with Llama-3.1 frequency scaling, sliding window, one sigmoid gate per head;
* mixer ``latent_attention`` — :class:`LatentSinkAttention`: queries straight from the input, a rotated key part shared by the heads
  (pairs ``(2i, 2i+1)``), sliding window; the cache row of a token is its normalised latent and the rotated part;
* mixer ``mlstm`` — :class:`RaggedMatrixMemoryMixer`;
* feed-forward ``dense`` — :class:`GatedMLP` (tanh GELU); ``moe`` — :class:`MoE`: biased fp32 router, softmax over the chosen logits, SiLU
  experts;
* output: final norm, head, ``logit_softcap * tanh(logits / logit_softcap)``.

Every size and constant comes from the checkpoint.  The engine side is the one the other hybrid stacks use: the paged cache with per-layer
shapes (:class:`LayeredBlockKVCacheManager`), state lines for everything carried per sequence, ragged rows (prompt portions beside single
decoded tokens) in one forward, decode steps replayed from CUDA graphs.
"""
from __future__ import annotations

import json
import os
from typing import List

import torch
import torch.nn as nn

from ... import ops
from ...config import InferenceConfig, NeuronConfig
from ...modules.attention.conv_window_attention import ConvWindowAttention
from ...modules.attention.latent_attention import LatentSinkAttention
from ...modules.checkpoint import stack_rows
from ...modules.kvcache import LayeredBlockKVCacheManager
from ...modules.mlp import GatedMLP
from ...modules.moe import ExpertMLPs, MoE, RouterTopK
from ...modules.norm import RMSNorm
from ...modules.rope import compute_inv_freq
from ...modules.sampling import Sampler
from ...modules.ssm import RaggedMatrixMemoryMixer
from ...parallel.layers import ColumnParallelLinear, ParallelEmbedding
from ..application_base import NeuronBaseForCausalLM
from ..fetodra.modeling_fetodra import NeuronFetodraModel
from ..model_base import PostNormDecoderLayer

MIXER_TYPES = ("attention", "latent_attention", "mlstm")


def rope_of(rot: dict):
    """(inverse frequencies fp64 [dims / 2], magnitude of cos / sin, cache tag) of a mixer's ``rot`` entry."""
    dims, base, sc = int(rot["dims"]), float(rot["base"]), rot.get("scaling")
    if not sc:
        return compute_inv_freq(dims, base, None, dtype=torch.float64)[0], 1.0, ("plain", dims, base)
    scaling = dict(rope_type="llama3", factor=sc["factor"], low_freq_factor=float(sc["low"]), high_freq_factor=float(sc["high"]),
                   original_max_position_embeddings=sc["original"])
    inv = compute_inv_freq(dims, base, scaling, dtype=torch.float64)[0]
    return inv, 1.0, ("llama3", dims, base, *(float(sc[k]) for k in ("factor", "low", "high", "original")))


class NavulornInferenceConfig(InferenceConfig):
    def get_required_attributes(self) -> List[str]:
        return ["layers", "norm", "postln_alpha", "vocab", "width"]

    def add_derived_config(self):
        self.num_cores_per_group = 1
        # names the engine's generic code looks up
        self.hidden_size, self.vocab_size, self.num_hidden_layers = self.width, self.vocab, len(self.layers)
        self.rms_norm_eps = float(self.norm["eps"])
        for name in ("embedding", "logit_softcap"):
            if not hasattr(self, name):
                setattr(self, name, None)
        self.embedding_scale = float((self.embedding or {}).get("scale", 1.0))
        self.bigram = (self.embedding or {}).get("bigram")
        for i, layer in enumerate(self.layers):
            if layer["type"] not in MIXER_TYPES:
                raise ValueError(f"layer {i}: unknown mixer type {layer['type']!r}")
            mlp = layer.get("mlp")
            if mlp is not None and mlp.get("kind") not in ("dense", "moe"):
                raise ValueError(f"layer {i}: unknown mlp kind {mlp.get('kind')!r}")
            m = layer["mixer"]
            if layer["type"] == "latent_attention" and int(m.get("rot_dim") or 0) and int(m["rot"]["dims"]) != int(m["rot_dim"]):
                raise ValueError(f"layer {i}: the rotation covers the whole rotated part (rot.dims == rot_dim)")

    @classmethod
    def get_neuron_config_cls(cls):
        return NeuronConfig

    @classmethod
    def from_pretrained(cls, model_path: str, neuron_config: NeuronConfig) -> "NavulornInferenceConfig":
        with open(os.path.join(model_path, "config.json")) as f:
            d = json.load(f)

        def load(self):
            for k, v in d.items():
                setattr(self, k, v)
        return cls(neuron_config, load_config=load)


class NeuronNavulornModel(NeuronFetodraModel):
    """The post-norm stack of :class:`NeuronFetodraModel` (ragged metadata, fp32 stream, final norm) with this design's parts."""
    design = "Navulorn"
    PREV_TOKEN = "prev_token"        # state line: the last token of a sequence

    def _mixer(self, i, spec, W, eps, dt, dev):
        m = spec["mixer"]
        kw = dict(eps=eps, layer_idx=i, dtype=dt, device=dev, tp_group=self.tp_group)
        heads, dim = m["heads"], m["dim"]
        vdim = m.get("vdim", dim)
        if spec["type"] == "mlstm":
            return RaggedMatrixMemoryMixer(W, heads, dim, vdim, float(m["gate_cap"]), **kw)
        window = (m.get("mask") or {}).get("size")
        rot_dim, rot = int(m.get("rot_dim") or 0), m.get("rot") or {}
        scale = float(m["scale"]) if m.get("scale") is not None else (dim + rot_dim) ** -0.5
        if spec["type"] == "latent_attention":
            return LatentSinkAttention(W, heads, dim, vdim, m["kv_rank"], scale=scale, sink=False, head_gate=False, rot_dim=rot_dim,
                                       rope=rope_of(rot) if rot_dim else None, rope_interleaved=True, window=window, **kw)
        dims = int(rot.get("dims") or 0)
        return ConvWindowAttention(W, heads, m.get("kv_heads", heads), dim, vdim, conv_taps=0, rot_dims=dims, rot_base=1.0,
                                   rope=rope_of(rot) if dims else None, rot_half=True, scale=scale, softcap=None, window=window, keep_first=0,
                                   bias=False, row_norm=True, out_gate="head", **kw)

    def _mlp(self, f, W, dt, dev):
        if f is None:
            return None
        if f["kind"] == "dense":
            return GatedMLP(W, f["ff"], "gelu_tanh", dt, False, self.tp_group, dev)
        r = f["router"]
        router = RouterTopK(r["experts"], r["top"], W, dt, "softmax", True, True, True, dev)
        return MoE(router, ExpertMLPs(r["experts"], W, f["expert"]["ff"], "silu", dt, False, dev))

    def init_model(self, config):
        nc = config.neuron_config
        dev, dt = self.device_, nc.torch_dtype
        W, eps = config.width, config.rms_norm_eps
        self.embed_tokens = ParallelEmbedding(config.vocab, W, None, dtype=dt, device=dev, shard_across_embedding=True, pad=True,
                                              tensor_model_parallel_group=self.tp_group)
        self.embed_bigrams = nn.Parameter(torch.zeros(int(config.bigram["buckets"]) + 1, W, dtype=dt, device=dev),
                                          requires_grad=False) if config.bigram else None
        norm = lambda: RMSNorm(W, eps, torch.float32, device=dev)       # noqa: E731
        layers = []
        for i, spec in enumerate(config.layers):
            mlp = self._mlp(spec.get("mlp"), W, dt, dev)
            layers.append(PostNormDecoderLayer(self._mixer(i, spec, W, eps, dt, dev), mlp, norm(), norm() if mlp is not None else None,
                                               config.postln_alpha, i))
        self.layers = nn.ModuleList(layers)
        self.norm = norm()
        self.lm_head = ColumnParallelLinear(W, config.vocab, bias=False, gather_output=False, dtype=dt, device=dev, pad=True,
                                            tensor_model_parallel_group=self.tp_group)

    def init_inference_optimization(self, config):
        nc = self.neuron_config
        if self.on_device_sampling:
            self.sampler = Sampler(nc, self.tp_group, vocab_shard=False)
        specs = {self.PREV_TOKEN: ((1,), torch.int32)} if self.embed_bigrams is not None else {}
        shapes = {}
        for i, layer in enumerate(self.layers):
            specs.update(layer.state_specs())
            if hasattr(layer.mixer, "kv_shape"):
                shapes[i] = layer.mixer.kv_shape()
        self.kv_mgr = LayeredBlockKVCacheManager(shapes, {}, nc.pa_num_blocks, nc.pa_block_size, nc.torch_dtype, self.device_,
                                                 state_specs=specs, num_slots=nc.kv_cache_batch_size, state_dtype=nc.torch_dtype)

    # ---- forward hooks ---------------------------------------------------------------------------------------------------
    def embed_step(self, input_ids, meta, inputs_embeds=None, vision_embeddings=None, vision_mask=None):
        ex, b = meta.extras, self.config.bigram or {}
        state = self.kv_mgr.states.tensor(self.PREV_TOKEN) if b else None
        h, lp = ops.bigram_embed(input_ids, self.embed_tokens.weight, self.embed_bigrams, self.config.embedding_scale,
                                 int(b.get("mul_prev", 0)), int(b.get("mul_cur", 0)), state, ex["state_lines"], ex["ctx_len"], ex["q_len"],
                                 ex["act_dtype"])
        ex["lp_stream"] = (h, lp)            # what the first layer's mixer reads
        return h

    def compute_logits(self, h):
        logits = super().compute_logits(h).float()
        cap = self.config.logit_softcap
        return float(cap) * torch.tanh(logits / float(cap)) if cap else logits


class NeuronNavulornForCausalLM(NeuronBaseForCausalLM):
    _model_cls = NeuronNavulornModel
    _STATE_DICT_MODEL_PREFIX = ""

    @classmethod
    def get_config_cls(cls):
        return NavulornInferenceConfig

    @classmethod
    def from_pretrained(cls, model_path: str, neuron_config: NeuronConfig):
        return cls(model_path, NavulornInferenceConfig.from_pretrained(model_path, neuron_config))

    @staticmethod
    def convert_hf_to_neuron_state_dict(sd: dict, config) -> dict:
        """Checkpoint names (``l<i>.mix.q`` ...) -> module parameters: the projections that read the same input stacked for one GEMM, the
        latent up-projections viewed per head, the experts' matrices stacked along a leading expert axis."""
        out = {"embed_tokens.weight": sd["embed"], "lm_head.weight": sd["head"], "norm.weight": sd["final.norm"]}
        if config.bigram:
            out["embed_bigrams"] = sd["bigram"]
        for i, spec in enumerate(config.layers):
            a, b = f"l{i}.", f"layers.{i}."
            out[b + "norm1.weight"] = sd[a + "norm1"]
            x, y, m = a + "mix.", b + "mixer.", spec["mixer"]
            parts = lambda *names: [sd[x + n] for n in names]          # noqa: E731
            if spec["type"] == "attention":
                out[y + "in_proj.weight"] = stack_rows(*parts("q", "k", "v", "g"))
                out[y + "q_norm_weight"], out[y + "k_norm_weight"] = sd[x + "q.norm"], sd[x + "k.norm"]
                out[y + "o_proj.weight"] = sd[x + "o"]
            elif spec["type"] == "latent_attention":
                H, R = m["heads"], m["kv_rank"]
                out[y + "in_proj.weight"] = torch.cat(parts("q", "dkv"), 0)
                out[y + "latent_norm_weight"] = sd[x + "dkv.norm"]
                out[y + "k_up"] = sd[x + "uk"].reshape(H, -1, R)
                out[y + "v_up"] = sd[x + "uv"].reshape(H, -1, R)
                out[y + "o_proj.weight"] = sd[x + "o"]
            else:
                out[y + "in_proj.weight"] = stack_rows(*parts("q", "k", "v", "g", "i", "f"))
                out[y + "i_bias"], out[y + "f_bias"] = sd[x + "i.b"], sd[x + "f.b"]
                out[y + "norm_weight"], out[y + "out_proj.weight"] = sd[x + "norm"], sd[x + "o"]
            f = spec.get("mlp")
            if f is None:
                continue
            out[b + "norm2.weight"] = sd[a + "norm2"]
            x, y = a + "mlp.", b + "mlp."
            if f["kind"] == "dense":
                out[y + "gate_up_proj.weight"] = torch.cat([sd[x + "gate"], sd[x + "up"]], 0)
                out[y + "down_proj.weight"] = sd[x + "down"]
            else:
                E = f["router"]["experts"]
                out[y + "router.linear_router.weight"], out[y + "router.linear_router.bias"] = sd[x + "router"], sd[x + "router.b"]
                out[y + "expert_mlps.gate_up_proj"] = torch.stack([torch.cat([sd[f"{x}e{e}.gate"], sd[f"{x}e{e}.up"]], 0) for e in range(E)], 0)
                out[y + "expert_mlps.down_proj"] = torch.stack([sd[f"{x}e{e}.down"] for e in range(E)], 0)
        return out

    def init_random_weights(self, seed: int = 0):
        """Benchmarks: N(0, 0.02) projections, unit norms, unbiased routers, forget gates that keep most of the memory."""
        super().init_random_weights(seed)
        with torch.no_grad():
            for name, p in self.model.named_parameters():
                if name.endswith(("norm1.weight", "norm2.weight", "norm_weight")) or name == "norm.weight":
                    p.fill_(1.0)
                elif name.endswith(("i_bias", "linear_router.bias")):
                    p.zero_()
                elif name.endswith("f_bias"):
                    p.fill_(4.0)
