"""The generic decoder: built from a ModelSpec, knows no architecture.

It owns the parts (embedding, one block per layer, final norm, head), says
which tensors it expects from a checkpoint, tells the cache manager what each
layer keeps, and runs one step: embed the step's tokens, run the layers in
the order the spec's ``schedule`` gives, gather the wanted rows, norm them and
project them to float32 logits (the reference computes the head for the last
row only in prefill, src/models/qwen2.cpp:2494-2499, and for every row in a
mixed batch, :1935-1945; here the caller says which rows).
"""
from __future__ import annotations

from typing import Dict, List, Optional, Tuple

import torch

from ..cache.manager import CacheManager
from ..config.model_spec import ModelSpec, PartSpec
from ..parts.base import (BLOCKS, EMBEDDINGS, FEED_FORWARDS, HEADS, MIXERS, NORMS, STREAM_STEPS, Block, BuildEnv,
                          LayerCache, ParamSpec, Part, StepContext, build_part)


class DecoderModel:
    def __init__(self, spec: ModelSpec, env: BuildEnv):
        spec.validate()
        self.spec = spec
        self.env = env
        self.embedding = build_part(EMBEDDINGS, spec.embedding, env)
        self.final_norm = build_part(NORMS, spec.final_norm, env)
        self.head = build_part(HEADS, spec.head, env)
        self.blocks: List[Block] = []
        # what runs right before a layer on each visit (None for most): a visit's own, also where the parts are borrowed
        self.entries: List[Optional[Part]] = [build_part(STREAM_STEPS, layer.entry, env) if layer.entry is not None else None
                                              for layer in spec.layers]
        for layer in spec.layers:
            if layer.weights_from is not None:
                # the same parts once more: parts hold weights only, what a layer keeps lives in its LayerCache
                self.blocks.append(self.blocks[layer.weights_from])
                continue
            mixer = build_part(MIXERS, layer.mixer, env)
            ffn = build_part(FEED_FORWARDS, layer.feed_forward, env) if layer.feed_forward is not None else None
            norm1 = build_part(NORMS, layer.mixer_norm, env)
            norm2 = build_part(NORMS, layer.ffn_norm, env) if layer.ffn_norm is not None else None
            block_class = BLOCKS.get(layer.block)
            if layer.block_params:
                self.blocks.append(block_class(mixer, ffn, norm1, norm2, env, params=dict(layer.block_params)))
            else:
                self.blocks.append(block_class(mixer, ffn, norm1, norm2, env))
        self.layer_caches: List[LayerCache] = [LayerCache() for _ in spec.layers]
        # single-token steps may be replayed from a CUDA graph only if every part says so
        self.graph_safe = all(part.graph_safe for _where, part, _spec in self.named_parts())

    # -- parameters -----------------------------------------------------------
    def named_parts(self) -> List[Tuple[str, Part, PartSpec]]:
        out: List[Tuple[str, Part, PartSpec]] = [("embedding", self.embedding, self.spec.embedding),
                                                 ("final_norm", self.final_norm, self.spec.final_norm),
                                                 ("head", self.head, self.spec.head)]
        for index, (block, layer) in enumerate(zip(self.blocks, self.spec.layers)):
            if self.entries[index] is not None:
                out.append((f"layers[{index}].entry", self.entries[index], layer.entry))
            if layer.weights_from is not None:
                continue
            out.append((f"layers[{index}].mixer_norm", block.mixer_norm, layer.mixer_norm))
            out.append((f"layers[{index}].mixer", block.mixer, layer.mixer))
            if block.ffn_norm is not None:
                out.append((f"layers[{index}].ffn_norm", block.ffn_norm, layer.ffn_norm))
            if block.feed_forward is not None:
                out.append((f"layers[{index}].feed_forward", block.feed_forward, layer.feed_forward))
        return out

    def manifest(self) -> Dict[str, Tuple[ParamSpec, str]]:
        """Checkpoint tensor name -> (what it must look like, where it is used)."""
        wanted: Dict[str, Tuple[ParamSpec, str]] = {}
        for where, part, spec in self.named_parts():
            for local, param in part.param_specs().items():
                if local not in spec.weights:
                    raise ValueError(f"{where}: the model spec names no tensor for parameter '{local}'")
                name = spec.weights[local]
                if name in wanted and (wanted[name][0].shape != param.shape or wanted[name][0].role != param.role):
                    raise ValueError(f"tensor '{name}' is wanted as {wanted[name][0]} by {wanted[name][1]} "
                                     f"and as {param} by {where}.{local}")
                wanted.setdefault(name, (param, f"{where}.{local}"))
        return wanted

    def load(self, tensors: Dict[str, torch.Tensor]) -> None:
        """Hands every part its parameters (``tensors`` is keyed by checkpoint name)."""
        for where, part, spec in self.named_parts():
            mine = {}
            for local, param in part.param_specs().items():
                name = spec.weights[local]
                if name in tensors:
                    mine[local] = tensors[name]
                elif not param.optional:
                    raise KeyError(f"{where}.{local}: tensor '{name}' was not loaded")
            if mine or part.param_specs():
                part.load(mine)
        for block, layer in zip(self.blocks, self.spec.layers):
            if layer.weights_from is None:
                block.loaded()

    def step_param_bytes(self, tokens: int = 1) -> int:
        """Bytes of parameters a step of ``tokens`` tokens reads: every part once per visit (a part whose share grows
        with the tokens says so through ``step_param_bytes``), the embedding rows not counted."""
        total = self.final_norm.param_bytes() + self.head.param_bytes()
        for index in self.spec.schedule:
            if self.entries[index] is not None:
                total += self.entries[index].param_bytes()
            for part in self.blocks[index].parts().values():
                grows = getattr(part, "step_param_bytes", None)
                total += grows(tokens) if grows is not None else part.param_bytes()
        return total

    # -- cache ----------------------------------------------------------------
    def declare_cache(self, manager: CacheManager) -> None:
        for index, (block, layer) in enumerate(zip(self.blocks, self.spec.layers)):
            if layer.cache_from is None:
                spec = block.mixer.cache_spec()
                for reader, other in zip(self.blocks, self.spec.layers):
                    # a layer that reads this one's entries may look further back than this one does
                    if other.cache_from == index and spec is not None and reader.mixer.cache_spec() is not None:
                        spec = spec.covering(reader.mixer.cache_spec())
                manager.add_layer(index, spec, block.mixer.state_spec(), block.mixer.extra_cache_specs())
            else:
                manager.add_layer(index, None, block.mixer.state_spec())

    def attach_cache(self, manager: CacheManager) -> None:
        self.layer_caches = [manager.layer_cache(index, source=layer.cache_from)
                             for index, layer in enumerate(self.spec.layers)]

    def cache_bytes_per_token(self) -> int:
        """Bytes of paged cache one token adds, over all layers that keep one (their ``cache_spec``)."""
        total = 0
        for block, layer in zip(self.blocks, self.spec.layers):
            spec = block.mixer.cache_spec() if layer.cache_from is None else None
            if spec is not None:
                for _name, shape in spec.entries:
                    count = 1
                    for extent in shape:
                        count *= int(extent)
                    total += count * self.env.dtype.itemsize
        return total

    def decode_cache_bytes(self, context: int) -> int:
        """Bytes of cache and state a single-token step moves for one request that holds ``context`` tokens, over the
        layers that keep their own (without windows, pooled entries or state: ``context * cache_bytes_per_token()``)."""
        return sum(block.mixer.decode_bytes(context) for block, layer in zip(self.blocks, self.spec.layers)
                   if layer.cache_from is None)

    def weight_bytes(self) -> int:
        """Bytes of all parameters on the device, a tensor that two parts share counted once."""
        total = 0
        for param, _where in self.manifest().values():
            count = 1
            for extent in param.shape:
                count *= max(int(extent), 0)
            total += count * (self.env.dtype.itemsize if param.role == "matrix" else 4)
        return total

    def step_flops(self, tokens: int, pairs: float, rows: int) -> float:
        """Floating-point operations of one step: ``tokens`` tokens through every scheduled layer, their queries
        meeting ``pairs`` (query, key) pairs per layer, and ``rows`` rows of logits."""
        total = self.head.flops(rows, 0.0)
        for index in self.spec.schedule:
            if self.entries[index] is not None:
                total += self.entries[index].flops(tokens, pairs)
            total += sum(part.flops(tokens, pairs) for part in self.blocks[index].parts().values())
        return total

    # -- one step -------------------------------------------------------------
    def forward(self, ctx: StepContext, logit_rows: Optional[torch.Tensor]) -> Optional[torch.Tensor]:
        """Runs the step's tokens through all layers; returns float32 logits [R, vocab] of the wanted rows."""
        x = self.embedding.forward(ctx.token_ids)
        schedule = self.spec.schedule
        # a stream step reads the embedding output: kept aside only if some layer has one
        x0 = x.clone() if any(self.entries[index] is not None for index in schedule) else None
        h = None                              # the next layer's first norm, when the previous layer produced it
        for step, index in enumerate(schedule):
            after = self.blocks[schedule[step + 1]] if step + 1 < len(schedule) else None
            if after is not None and self.entries[schedule[step + 1]] is not None:
                after = None                  # the stream changes before the next layer: nothing of it can be normed ahead
            following = after.mixer_norm if after is not None else None
            block = self.blocks[index]
            if self.entries[index] is not None:
                self.entries[index].forward(x, x0, ctx)
            more = ({"next_takes_deferred": after is not None and after.mixer.takes_deferred_rows}
                    if block.passes_deferred_rows else {})
            h = block.forward(x, ctx, self.layer_caches[index], h=h, next_norm=following, **more)
        if logit_rows is None or logit_rows.numel() == 0:
            return None
        h = self.final_norm.forward(x, rows=logit_rows)
        return self.head.forward(h)
