"""A decoder as data: an embedding, a list of layers, the ORDER in which layers run, a final
norm and an output head.  The model builder of an architecture fills a `ModelSpec` from its
configuration; `DecoderModel` builds the parts and runs a step.  Nothing here knows an
architecture's name.

The order is a list of `ScheduleEntry`: which layer runs, which cache it uses and whether it
appends to it.  The default is each layer once with a cache of its own; a list may name a layer
twice (with a second cache) or let a layer read a cache that an earlier entry wrote.
"""
from __future__ import annotations

from dataclasses import dataclass, field
from typing import Optional

import torch

from ..parts import ARRANGEMENTS, JUNCTIONS, NORMS, PartSpec, build_layer, check_layer, layer_tensor_specs, lookup, MIXERS
from ..parts.linear import STORE, linear, prepare_weight
from ..weights import TensorSpec


@dataclass(frozen=True)
class ScheduleEntry:
    layer: int
    cache: Optional[int] = None     # id of the cache this entry uses (None: the mixer has none)
    writes: bool = True             # False: read a cache that another entry fills


@dataclass
class ModelSpec:
    hidden_size: int
    vocab_size: int
    max_positions: Optional[int]                    # None: the design has no limit of its own
    layers: list
    final_norm: PartSpec
    schedule: list = field(default_factory=list)
    embedding_scale: float = 1.0
    logit_scale: float = 1.0
    embedding_name: str = "model.embed_tokens.weight"
    head_name: Optional[str] = "lm_head.weight"     # None: tied to the embedding table
    layer_prefix: str = "model.layers.{}."
    final_norm_prefix: str = "model.norm."
    eos_token_ids: tuple = ()
    position_table_name: Optional[str] = None       # a learned vector per position [max_positions, hidden], added to the embedding
    sinusoidal_base: Optional[float] = None         # a sinusoidal vector of the position is added to the embedding: sine of p * base^(-2i/hidden) in column 2i, cosine in 2i + 1
    junctions: dict = field(default_factory=dict)   # schedule position -> PartSpec of a junction that runs ahead of that entry
    streams: int = 1                                # copies of the residual stream in a token's row (hyper-connections); all start as the embedding output, their sum goes to the final norm
    logit_softcap: Optional[float] = None           # logits <- cap * tanh(logits / cap)

    def __post_init__(self):
        if not self.schedule:
            self.schedule = [
                ScheduleEntry(i, i if self._mixer(i).cache_request(self.layers[i].mixer.params) else None)
                for i in range(len(self.layers))]
        for entry in self.schedule:
            if not 0 <= entry.layer < len(self.layers):
                raise ValueError(f"schedule names layer {entry.layer}, the model has {len(self.layers)}")
        for layer in self.layers:
            check_layer(layer)                      # a size that a part or its kernels cannot take is refused here
            if lookup(ARRANGEMENTS, layer.arrangement, "arrangement").streams(layer) != self.streams:
                raise ValueError(f"the model keeps {self.streams} residual streams; a layer's arrangement keeps another number")
        if self.streams != 1 and self.junctions:
            raise ValueError("junctions act on a single residual stream")
        if self.sinusoidal_base is not None and (not float(self.sinusoidal_base) > 0 or self.position_table_name is not None or
                                                 self.streams != 1):
            raise ValueError("sinusoidal_base must be positive, without a position table and with a single residual stream")
        if self.logit_softcap is not None and not float(self.logit_softcap) > 0:
            raise ValueError("logit_softcap must be positive")
        for position, junction in self.junctions.items():
            if not 0 <= position < len(self.schedule):
                raise ValueError(f"a junction is attached to schedule position {position}, the schedule has {len(self.schedule)}")
            lookup(JUNCTIONS, junction.kind, "junction").check_params(junction.params)
        requests = {}
        writers = set()
        for entry in self.schedule:
            request = self._mixer(entry.layer).cache_request(self.layers[entry.layer].mixer.params)
            if (request is None) != (entry.cache is None):
                raise ValueError(f"schedule entry {entry}: the mixer's cache need and the entry disagree")
            if entry.cache is None:
                continue
            if requests.setdefault(entry.cache, request) != request:
                raise ValueError(f"cache {entry.cache} is shared by layers with different needs")
            if entry.writes:
                if entry.cache in writers:
                    raise ValueError(f"cache {entry.cache} is written by two schedule entries")
                writers.add(entry.cache)
            elif entry.cache not in writers:
                raise ValueError(f"cache {entry.cache} is read before any entry writes it")

    def _mixer(self, layer: int):
        return lookup(MIXERS, self.layers[layer].mixer.kind, "mixer")

    def tensor_specs(self) -> list:
        specs = [TensorSpec(self.embedding_name, (self.vocab_size, self.hidden_size))]
        if self.position_table_name is not None:
            specs.append(TensorSpec(self.position_table_name, (self.max_positions, self.hidden_size)))
        seen = set()
        for position in sorted(self.junctions):
            junction = self.junctions[position]
            for spec in lookup(JUNCTIONS, junction.kind, "junction").tensor_specs(junction.params, ""):
                if spec.name not in seen:             # junctions may share tensors (one weight for every pass)
                    seen.add(spec.name)
                    specs.append(spec)
        for i, layer in enumerate(self.layers):
            specs += layer_tensor_specs(layer, self.layer_prefix.format(i))
        specs += lookup(NORMS, self.final_norm.kind, "norm").tensor_specs(self.final_norm.params,
                                                                           self.final_norm_prefix)
        if self.head_name is not None:
            specs.append(TensorSpec(self.head_name, (self.vocab_size, self.hidden_size)))
        return specs

    def cache_requests(self) -> dict:
        """cache id -> KVCacheRequest."""
        out = {}
        for entry in self.schedule:
            if entry.cache is not None:
                out[entry.cache] = self._mixer(entry.layer).cache_request(self.layers[entry.layer].mixer.params)
        return out

    def state_requests(self) -> dict:
        """state id -> StateRequest: the schedule position for a mixer that keeps per-request state, ("layer",
        schedule position) for an arrangement that does.  A layer that runs twice has a state for each run."""
        out = {}
        for position, entry in enumerate(self.schedule):
            layer = self.layers[entry.layer]
            request = self._mixer(entry.layer).state_request(layer.mixer.params)
            if request is not None:
                out[position] = request
            request = lookup(ARRANGEMENTS, layer.arrangement, "arrangement").state_request(layer)
            if request is not None:
                out[("layer", position)] = request
        return out


class DecoderModel:
    def __init__(self, spec: ModelSpec, tensors: dict, runtime):
        self.spec, self.runtime = spec, runtime
        device = runtime.device

        def on_device(names):
            return {n: tensors[n].to(device) for n in names if n in tensors}      # (an optional tensor may be absent)

        table = tensors[spec.embedding_name].to(device)
        self.embedding = prepare_weight(table, runtime)
        self.position_table = None
        if spec.position_table_name is not None:
            self.position_table = prepare_weight(tensors[spec.position_table_name].to(device), runtime)
        self.position_frequencies = None
        if spec.sinusoidal_base is not None:
            exponents = -2.0 * torch.arange((spec.hidden_size + 1) // 2, dtype=torch.float64) / spec.hidden_size
            self.position_frequencies = (float(spec.sinusoidal_base) ** exponents).to(torch.float32).to(device)
        self.junctions = {}
        for position, junction in spec.junctions.items():
            cls = lookup(JUNCTIONS, junction.kind, "junction")
            names = [s.name for s in cls.tensor_specs(junction.params, "")]
            self.junctions[position] = cls(junction.params, on_device(names), "", runtime)
        self._keeps_first = any(j.needs_first for j in self.junctions.values())
        self.layers = []
        for i, layer in enumerate(spec.layers):
            prefix = spec.layer_prefix.format(i)
            names = [s.name for s in layer_tensor_specs(layer, prefix)]
            self.layers.append(build_layer(layer, on_device(names), prefix, runtime))
        norm_cls = lookup(NORMS, spec.final_norm.kind, "norm")
        names = [s.name for s in norm_cls.tensor_specs(spec.final_norm.params, spec.final_norm_prefix)]
        self.final_norm = norm_cls(spec.final_norm.params, on_device(names), spec.final_norm_prefix, runtime)
        record = self.final_norm.rms_record()
        self._final_weight = record[0].to(torch.float32).contiguous() if record is not None else None
        if spec.head_name is None:
            self.head = self.embedding
        else:
            self.head = prepare_weight(tensors[spec.head_name].to(device), runtime)
        # layers of one description launch alike: one of each answers for all when a step's graph key is made
        distinct = {}
        for layer_spec, layer in zip(spec.layers, self.layers):
            distinct.setdefault(repr(layer_spec), layer)
        self._key_layers = list(distinct.values()) + [self.final_norm] + list(self.junctions.values())
        self._own_state = [lookup(ARRANGEMENTS, spec.layers[entry.layer].arrangement, "arrangement").state_request(
            spec.layers[entry.layer]) is not None for entry in spec.schedule]
        # decode steps may be captured in CUDA graphs only if every part launches the same way each step
        self.graph_safe = (all(layer.graph_safe for layer in self.layers) and bool(self.final_norm.graph_safe)
                           and all(j.graph_safe for j in self.junctions.values()))

    def graph_key(self, ctx) -> tuple:
        """What a captured step is good for: the step's numbers of tokens, of wanted rows, of single-token entries
        and of portions, its context bucket, and whatever else of its shape the parts say their launches depend on
        (each distinct answer once)."""
        seen, extra = set(), []
        for layer in self._key_layers:
            key = layer.graph_key(ctx)
            if key and key not in seen:
                seen.add(key)
                extra.append(key)
        return (ctx.n_tokens, ctx.n_out, ctx.context_bucket, ctx.n_single, ctx.n_prefill_segments, tuple(extra))

    def forward(self, ctx) -> torch.Tensor:
        """Run the step described by `ctx`; returns 32-bit logits [ctx.n_out, vocab] (device).  When fewer rows
        are wanted than the step brings, the last entry of the schedule is told which (an arrangement that can
        then computes only what those rows need and hands back their residual rows; the reference's pruning of
        the last layer, src/inference/llama_fusion.rs:45-60, src/gpu/kernels/llama.rs:185-198)."""
        rt, spec = self.runtime, self.spec
        n = ctx.n_tokens
        streams = spec.streams
        h = ctx.buffer("model.h", (n, streams * spec.hidden_size), torch.float32)
        first = ctx.buffer("model.h0", (n, spec.hidden_size), torch.float32) if self._keeps_first else None
        rounded = None
        if streams > 1:
            if self.position_table is not None:
                raise ValueError("a position table with several residual streams is not built")
            rt.ops.embedding_streams(ctx.tokens, self.embedding, h, streams, spec.embedding_scale, ctx.error_flag)
        elif self.position_frequencies is not None:
            # (a first layer that reads the stream itself gets it in the compute element type from the same kernel)
            if rt.compute_dtype != torch.float32 and self.layers[spec.schedule[0].layer].reads_stream:
                rounded = ctx.buffer("block.x", (n, spec.hidden_size), rt.compute_dtype)
            rt.ops.embedding_sinusoidal(ctx.tokens, ctx.positions, self.embedding, self.position_frequencies, h,
                                        spec.embedding_scale, copy=rounded, error_flag=ctx.error_flag)
            if first is not None:
                first.copy_(h)
        elif self.position_table is not None:
            rt.ops.embedding_positions(ctx.tokens, ctx.positions, self.embedding, self.position_table, h,
                                       spec.embedding_scale, copy=first, error_flag=ctx.error_flag)
        else:
            rt.ops.embedding(ctx.tokens, self.embedding, h, spec.embedding_scale, ctx.error_flag, copy=first)
        ctx.rounded_stream = rounded
        picked = None
        last = len(spec.schedule) - 1
        for position, entry in enumerate(spec.schedule):
            junction = self.junctions.get(position)
            owed = getattr(ctx, "owed", None)
            if owed is not None and (junction is not None or type(self.layers[entry.layer]) is not type(owed[0])):
                owed[0].settle(ctx, h)
            if junction is not None:
                junction.forward(ctx, h, first)
                ctx.rounded_stream = None
            kv = ctx.kv_view(entry.cache, entry.writes) if entry.cache is not None else None
            layer = self.layers[entry.layer]
            more = {"own_state": ctx.state(("layer", position))} if self._own_state[position] else {}
            if position == last and ctx.n_out < n and getattr(layer, "supports_rows", False):
                picked = layer.forward(ctx, h, kv=kv, state=ctx.state(position), rows=ctx.out_rows, n_rows=ctx.n_out, **more)
            else:
                layer.forward(ctx, h, kv=kv, state=ctx.state(position), **more)
            if not getattr(layer, "reads_stream", False):
                ctx.rounded_stream = None
        owed = getattr(ctx, "owed", None)
        if owed is not None:
            if ctx.n_out > 0:
                owed[0].settle(ctx, h)          # (without wanted rows nobody reads the stream again)
            ctx.owed = None
        if ctx.n_out == 0:
            return ctx.logits_buffer(0, spec.vocab_size)
        y = ctx.buffer("model.y", (ctx.n_out, spec.hidden_size), rt.compute_dtype)
        if streams > 1:
            # the wanted rows' streams are added up, and normed in the same pass where the final norm is an RMS norm
            total = ctx.buffer("model.sum", (ctx.n_out, spec.hidden_size), torch.float32)
            record = self.final_norm.rms_record()
            if record is not None:
                rt.ops.hyper_step(h, streams, rows_index=ctx.out_rows, u=total, norm_weight=self._final_weight, normed=y,
                                  eps=record[1])
            else:
                rt.ops.hyper_step(h, streams, rows_index=ctx.out_rows, u=total)
                self.final_norm.forward(ctx, total, y)
        elif picked is not None:
            self.final_norm.forward(ctx, picked, y)
        else:
            self.final_norm.forward(ctx, h, y, rows_index=ctx.out_rows)
        logits = ctx.logits_buffer(ctx.n_out, spec.vocab_size)
        linear(rt, STORE, y, self.head, logits, spec.logit_scale, error_flag=ctx.error_flag, name="head")
        if spec.logit_softcap is not None:
            rt.ops.softcap_rows(logits, float(spec.logit_softcap))
        return logits
