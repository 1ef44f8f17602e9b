"""The model: an embedding, the layers a `ModelSpec` lists, run in the order of
its schedule, a final norm and the output product.

gpt-fast's `Transformer` (model.py:102-150) hard-wires one kind of block and
computes logits for every position; this one is built from the spec's parts,
runs a packed batch of sequences of unequal lengths against the paged cache
and computes logits only for the rows that are asked for.  It knows no
architecture: everything specific came in through the spec.
"""
from typing import Dict, Optional

import torch

from .. import ops
from ..cache import Cache, CacheNeeds, EntryView
from ..config.spec import ModelSpec, PartSpec
from ..ops.types import BatchMeta
from ..parts.residual import Residual
from ..parts.streams import Streams
from ..parts import EMBEDDINGS, JUNCTIONS, NORMS, POSITIONS, build_block, build_part
from ..weights.loader import ParamSpec

EMBEDDING_CACHE_ENTRY = -1        # the cache entry of the embedding part's per-sequence state (layers count from 0)

COMPUTE_DTYPES = {"bfloat16": torch.bfloat16, "bf16": torch.bfloat16, "float32": torch.float32, "fp32": torch.float32}


def compute_dtype(dtype) -> torch.dtype:
    if isinstance(dtype, torch.dtype):
        if dtype not in (torch.bfloat16, torch.float32):
            raise ValueError(f"the model runs in bfloat16 or float32, not {dtype}")
        return dtype
    if dtype not in COMPUTE_DTYPES:
        raise ValueError(f"unknown dtype '{dtype}' (bfloat16 or float32)")
    return COMPUTE_DTYPES[dtype]


class Transformer:
    def __init__(self, spec: ModelSpec, dtype=torch.bfloat16, device="cuda"):
        spec.validate()
        self.spec = spec
        self.dtype = compute_dtype(dtype)
        self.device = torch.device(device)
        self.dim, self.vocab_size = spec.dim, spec.vocab_size

        positions = []                             # (PartSpec, object): one object per distinct spec

        def position_for(ps: Optional[PartSpec]):
            if ps is None:
                return None
            for known, obj in positions:
                if known is ps or known == ps:
                    return obj
            obj = build_part(POSITIONS, ps)
            positions.append((ps, obj))
            return obj

        self.blocks = [build_block(ls, spec.dim, self.dtype, position_for(ls.position)) for ls in spec.layers]
        self.positions = [obj for _, obj in positions]
        if any(getattr(b, "takes_streams", False) != bool(spec.streams) for b in self.blocks):
            raise ValueError("a model with several residual streams is made of blocks that take streams, any other model of blocks that do not")
        self.final_norm = build_part(NORMS, spec.final_norm, dtype=self.dtype)
        self.embedding = None if spec.embedding is None else build_part(EMBEDDINGS, spec.embedding, dtype=self.dtype)
        self.junctions = [build_part(JUNCTIONS, ps, dtype=self.dtype) for ps in spec.junctions]
        self.embed_weight = None
        self.head_weight = None
        self.token_table = None            # [vocab, spec.token_table]: what token inputs read of a token
        self.after_layer = None            # a callable(stream) run behind every layer of a step (tests look at the stream)

    # ---- parameters -------------------------------------------------------------
    def param_specs(self) -> Dict[str, ParamSpec]:
        specs = {"embed.weight": ParamSpec((self.vocab_size, self.dim)),
                 "head.weight": ParamSpec((self.vocab_size, self.dim))}
        for name, s in self.final_norm.param_specs().items():
            specs[f"final_norm.{name}"] = s
        if self.embedding is not None:
            for name, s in self.embedding.param_specs().items():
                specs[f"embedding.{name}"] = s
        if self.spec.token_table:
            specs["token_table.weight"] = ParamSpec((self.vocab_size, self.spec.token_table))
        for i, j in enumerate(self.junctions):
            for name, s in j.param_specs().items():
                specs[f"junctions.{i}.{name}"] = s
        for i, b in enumerate(self.blocks):
            for pname, part in b.parts().items():
                for name, s in part.param_specs().items():
                    specs[f"layers.{i}.{pname}.{name}"] = s
        return specs

    def load_params(self, tensors: Dict[str, torch.Tensor]) -> None:
        """Hand every part its tensors (as named by `param_specs`)."""
        want = self.param_specs()
        missing = sorted(set(want) - set(tensors))
        if missing:
            raise KeyError(f"model parameters without a tensor: {missing}")
        for name, s in want.items():
            if tuple(tensors[name].shape) != tuple(s.shape):
                raise ValueError(f"parameter {name}: expected shape {tuple(s.shape)}, got {tuple(tensors[name].shape)}")

        def sub(prefix):
            return {k[len(prefix):]: v for k, v in tensors.items() if k.startswith(prefix)}
        self.embed_weight = tensors["embed.weight"]
        self.head_weight = tensors["head.weight"]
        if self.spec.tie_embeddings and self.head_weight.data_ptr() != self.embed_weight.data_ptr():
            raise ValueError("the spec ties the output to the embedding, but two tensors were given")
        self.final_norm.load(sub("final_norm."))
        if self.embedding is not None:
            self.embedding.load(sub("embedding."))
        for i, j in enumerate(self.junctions):
            j.load(sub(f"junctions.{i}."))
        self.token_table = tensors.get("token_table.weight")
        for i, b in enumerate(self.blocks):
            for pname, part in b.parts().items():
                part.load(sub(f"layers.{i}.{pname}."))
                if hasattr(part, "bind_token_table"):
                    part.bind_token_table(self.token_table)

    def export_params(self) -> Dict[str, torch.Tensor]:
        """Every parameter under the name and in the layout of `param_specs` (the inverse of `load_params`);
        each part gives its own back through `export()`."""
        out = {"embed.weight": self.embed_weight, "head.weight": self.head_weight}
        for name, t in self.final_norm.export().items():
            out[f"final_norm.{name}"] = t
        if self.embedding is not None:
            for name, t in self.embedding.export().items():
                out[f"embedding.{name}"] = t
        if self.token_table is not None:
            out["token_table.weight"] = self.token_table
        for i, j in enumerate(self.junctions):
            for name, t in j.export().items():
                out[f"junctions.{i}.{name}"] = t
        for i, b in enumerate(self.blocks):
            for pname, part in b.parts().items():
                if not hasattr(part, "export"):
                    raise NotImplementedError(f"part '{pname}' of layer {i} ({type(part).__name__}) has no export()")
                for name, t in part.export().items():
                    out[f"layers.{i}.{pname}.{name}"] = t
        return out

    def graph_safe(self) -> bool:
        """Whether a step of this model may be captured in a CUDA graph: every part launches kernels only.  A part
        that reads device values on the host says so with `graph_safe = False`."""
        parts = [self.final_norm] + [p for b in self.blocks for p in b.parts().values()] + list(self.positions) + self.junctions
        if self.embedding is not None:
            parts.append(self.embedding)
        return all(getattr(p, "graph_safe", True) for p in parts + list(self.blocks))

    def weight_bytes(self, with_embedding=False) -> int:
        """Bytes of the parameters a decode step streams (every matrix once)."""
        seen, total = set(), 0

        def add(t):
            nonlocal total
            if t is not None and t.data_ptr() not in seen:
                seen.add(t.data_ptr())
                total += t.numel() * t.element_size()
        add(self.head_weight)
        if self.token_table is not None:
            seen.add(self.token_table.data_ptr())          # a row per token, not the table
        if with_embedding:
            add(self.embed_weight)
        for e in self.spec.schedule:
            for part in self.blocks[e.layer].parts().values():
                for v in vars(part).values():
                    if isinstance(v, torch.Tensor):
                        add(v)
        for part in self.junctions:
            for v in vars(part).values():
                if isinstance(v, torch.Tensor):
                    add(v)
        for v in vars(self.final_norm).values():
            if isinstance(v, torch.Tensor):
                add(v)
        return total

    # ---- cache ---------------------------------------------------------------------
    def cache_needs(self) -> Dict[int, CacheNeeds]:
        needs = {}
        if self.embedding is not None:
            needs[EMBEDDING_CACHE_ENTRY] = self.embedding.cache_needs()
        for e in self.spec.schedule:
            if e.owns_cache:
                needs[e.cache] = self.blocks[e.layer].cache_needs()
        return needs

    def new_cache(self, max_tokens: int, max_seqs: Optional[int] = None, max_seq_len: Optional[int] = None,
                  page_size: Optional[int] = None) -> Cache:
        limit = self.spec.max_position or None
        if max_seq_len is None:
            max_seq_len = limit
        elif limit and max_seq_len > limit:
            raise ValueError(f"max_seq_len {max_seq_len} exceeds the model's longest sequence {limit}")
        kw = {} if page_size is None else {"page_size": page_size}
        cache = Cache(self.cache_needs(), self.dtype, self.device, max_tokens=max_tokens, max_seqs=max_seqs,
                      max_seq_len=max_seq_len, **kw)
        for p in self.positions:
            p.prepare(cache.max_pages * cache.page_size, self.device)
        return cache

    def default_cache(self, max_tokens: int, max_seqs: int, max_seq_len: int) -> Cache:
        """The cache `generate` uses when none is given: kept between calls and replaced only when a
        call needs more tokens, sequences or length than it has (gpt-fast's setup_caches grows the
        same way, model.py:117-119)."""
        c = getattr(self, "_default_cache", None)
        if (c is None or c.n_pages * c.page_size < max_tokens or c.n_slots < max_seqs or c.max_seq_len < max_seq_len
                or c.slots.n_free != c.n_slots):
            self._default_cache = None            # let the old pools go before the new ones are made
            c = self.new_cache(max_tokens, max_seqs=max_seqs,
                               max_seq_len=min(max(max_seq_len, 1), self.spec.max_position or max_seq_len))
            self._default_cache = c
        return c

    # ---- one step ------------------------------------------------------------------------
    def forward(self, tokens: torch.Tensor, batch: BatchMeta, cache: Cache,
                want_rows: Optional[torch.Tensor], n_want: Optional[int] = None) -> torch.Tensor:
        """tokens int32 [T] (packed) -> float32 logits [W, V] at the packed rows
        `want_rows` (int32 [W]); None wants every row.  Appends this step's keys
        and values to the cache; the caller advances the lengths afterwards."""
        T = batch.n_tokens
        ops.set_launch_overlap(self.spec.launch_overlap)
        batch.tokens = tokens
        x = torch.empty(T, self.dim, dtype=torch.float32, device=self.device)
        scale = 1.0 if self.spec.embed_scale is None else float(self.spec.embed_scale)
        if self.embedding is None:
            ops.embed(tokens, self.embed_weight, x, batch.status, scale)
        else:
            self.embedding.forward(tokens, self.embed_weight, x, batch, cache.view(EMBEDDING_CACHE_ENTRY), scale)
        x0 = x                                  # the embedding output, which junctions read again
        if self.junctions and self.spec.schedule[0].junction is None:
            x = x0.clone()                      # layers ahead of the first junction write into the stream
        x = Streams(x, self.spec.streams) if self.spec.streams else Residual(x)
        for e in self.spec.schedule:
            if e.junction is not None:
                self.junctions[e.junction].forward(x, x0, e.turn)
            if e.kv_from is None:
                self.blocks[e.layer].forward(x, batch, cache.view(e.cache), append=e.owns_cache)
            else:
                # another entry's keys and values, the run's own state
                view = EntryView(kv=cache.view(e.kv_from).kv, state=cache.view(e.cache).state)
                self.blocks[e.layer].forward(x, batch, view, append=False)
            if self.after_layer is not None:
                self.after_layer(x)
        W = T if want_rows is None else (n_want if n_want is not None else want_rows.shape[0])
        logits = torch.empty(W, self.vocab_size, dtype=torch.float32, device=self.device)
        if W:
            h = torch.empty(W, self.dim, dtype=self.dtype, device=self.device)
            self.final_norm.forward(x.total() if self.spec.streams else x, h, want_rows)
            ops.linear(h, self.head_weight, logits)
            if self.spec.logit_cap is not None:
                ops.softcap(logits, float(self.spec.logit_cap))
        return logits
