"""A decoder put together from a :class:`~pylon_b200.parts.spec.ModelSpec`.

Embedding, the layers in their run order, final norm and vocabulary head.  The class knows
no architecture: which parts a layer has, their sizes and the order of the runs all come
from the spec.  The data flow is raun6k/Pylon's packed forward
(src/pylon/model/model.py:124-144): embed, blocks, then norm and head only at the rows
whose logits are wanted.  Two things architectures do around that flow are constants of the
spec: a factor on the embedding rows, and a factor and a soft cap on the logits.
"""
from __future__ import annotations

from typing import Callable, Mapping, Optional, Sequence

import torch

from pylon_b200.kernels import ops
from pylon_b200.parts.base import BLOCKS, NORMS, CacheNeed, LayerCache, ResidualStream, StepView, TensorDecl
from pylon_b200.parts.spec import ModelSpec

_ROLE_DTYPES = {"vector": torch.float32, "table": torch.int32}


class DecoderModel:
    def __init__(self, spec: ModelSpec) -> None:
        self.spec = spec
        self.blocks = [BLOCKS.build(layer.block) for layer in spec.layers]
        self.final_norm = NORMS.build(spec.final_norm)
        self.embedding_norm = None if spec.embedding_norm is None else NORMS.build(spec.embedding_norm)
        self.embedding: Optional[torch.Tensor] = None
        self.lm_head: Optional[torch.Tensor] = None
        self.position_table: Optional[torch.Tensor] = None   # learnt vectors per position, added to the embedding rows
        self.reentry: Optional[torch.Tensor] = None          # [width, 2 width]: how a run with ``reenter`` is entered
        self.dtype: Optional[torch.dtype] = None
        self.device: Optional[torch.device] = None

    # -- weights -------------------------------------------------------------------------
    def tensor_decls(self) -> dict[str, TensorDecl]:
        """Every checkpoint tensor the model needs, by full name."""
        spec = self.spec
        decls = {spec.embedding_name: TensorDecl(spec.embedding_name, (spec.vocab_size, spec.width))}
        if spec.lm_head_name is not None:
            decls[spec.lm_head_name] = TensorDecl(spec.lm_head_name, (spec.vocab_size, spec.width))
        if spec.position_name is not None:
            decls[spec.position_name] = TensorDecl(spec.position_name, (spec.position_rows, spec.width))
        if spec.reentry_name is not None:
            decls[spec.reentry_name] = TensorDecl(spec.reentry_name, (spec.width, 2 * spec.width), "matrix", (0.0, (2 * spec.width) ** -0.5))
        for decl in self.final_norm.tensors():
            name = spec.final_norm_prefix + decl.name
            decls[name] = TensorDecl(name, decl.shape, decl.role, decl.init)
        if self.embedding_norm is not None:
            for decl in self.embedding_norm.tensors():
                name = spec.embedding_norm_prefix + decl.name
                decls[name] = TensorDecl(name, decl.shape, decl.role, decl.init)
        for layer, block in zip(spec.layers, self.blocks):
            for decl in block.tensors():
                name = layer.prefix + decl.name
                if name in decls:
                    raise ValueError(f"two parts declare the tensor '{name}'")
                decls[name] = TensorDecl(name, decl.shape, decl.role, decl.init)
        return decls

    def load(self, fetch: Callable[[str], torch.Tensor], dtype: torch.dtype, device: torch.device) -> None:
        """``fetch(name)`` returns a checkpoint tensor as stored (host memory).  Tensors are
        moved part by part so that host and device never hold a second copy of the model."""
        self.dtype, self.device = dtype, torch.device(device)

        def place(decl: TensorDecl) -> torch.Tensor:
            target = _ROLE_DTYPES.get(decl.role, dtype)
            return fetch(decl.name).to(device=self.device, dtype=target)

        spec = self.spec
        decls = self.tensor_decls()
        self.embedding = place(decls[spec.embedding_name]).contiguous()
        self.lm_head = self.embedding if spec.lm_head_name is None else place(decls[spec.lm_head_name]).contiguous()
        if spec.position_name is not None:
            self.position_table = place(decls[spec.position_name]).contiguous()
        if spec.reentry_name is not None:
            self.reentry = place(decls[spec.reentry_name]).contiguous()
        self.final_norm.load(
            {decl.name: place(decls[spec.final_norm_prefix + decl.name]) for decl in self.final_norm.tensors()}, dtype, self.device
        )
        if self.embedding_norm is not None:
            self.embedding_norm.load(
                {decl.name: place(decls[spec.embedding_norm_prefix + decl.name]) for decl in self.embedding_norm.tensors()}, dtype, self.device
            )
        for layer, block in zip(spec.layers, self.blocks):
            block.load({decl.name: place(decls[layer.prefix + decl.name]) for decl in block.tensors()}, dtype, self.device)

    def weight_bytes(self) -> int:
        """Bytes of weights one step reads (each layer once per run; the head once)."""
        total = self.lm_head.numel() * self.lm_head.element_size() + self.final_norm.weight_bytes()
        for run in self.spec.order:
            total += self.blocks[run.layer].weight_bytes()
            if run.reenter:
                total += self.reentry.numel() * self.reentry.element_size()
        return total

    def takes_padding(self) -> bool:
        """Whether every layer that runs is right for steps padded to the size of a captured graph."""
        return all(self.blocks[run.layer].takes_padding for run in self.spec.order)

    # -- cache ---------------------------------------------------------------------------
    def cache_needs(self) -> list[Optional[CacheNeed]]:
        """Per run of the order: what its mixer keeps between steps (``None`` where the run
        reads another run's cache)."""
        return [
            None if run.cache_of is not None else self.blocks[run.layer].mixer.cache_need()
            for run in self.spec.order
        ]

    # -- run -----------------------------------------------------------------------------
    def forward(self, step: StepView, caches: Sequence[LayerCache], taps: Optional[list] = None) -> Optional[torch.Tensor]:
        """Runs the step's tokens; returns float32 logits ``[num_logits, vocab]`` at
        ``step.logit_rows`` (``None`` when no logits are wanted: the head is skipped).
        ``caches[i]`` belongs to run ``i`` of the order (a shared cache appears twice).
        ``taps``: a list that receives the residual stream after every run, float32 ``[T, width]``
        (the sum of the copies where the model keeps several) - for looking at a model layer by layer."""
        step.carry = {}
        if self.embedding_norm is not None:   # the normed rows are the stream: one kernel, which leaves it in the compute dtype as well
            stream = self.embedding_norm.enter(step.token_ids, self.embedding, self.spec.embedding_scale)
        else:
            stream = ResidualStream(ops.embed_gather(step.token_ids, self.embedding, scale=self.spec.embedding_scale, copies=self.spec.streams))
        residual = stream.residual
        if self.position_table is not None:   # the learnt vector of each token's position joins its embedding row, in 32-bit like the sum
            ops.embed_gather(step.positions, self.position_table, out=residual, copies=self.spec.streams, accumulate=True)
        entered = residual.clone() if self.reentry is not None else None   # the embedding output, for the runs that re-enter
        for position, run in enumerate(self.spec.order):
            if run.reenter:
                # x <- W [x; x0]: what is pending joins the sum, both halves are laid side by side in the compute dtype, and the
                # product's 32-bit result is the new sum
                stream.flush()
                stream.residual = ops.linear(ops.concat_cast(stream.residual, entered, self.dtype), self.reentry, out_dtype=torch.float32)
            if run.add_embedding:
                stream.flush()   # what the run before left pending joins the sum first; then the embedding rows, in 32-bit like the sum itself
                ops.embed_gather(step.token_ids, self.embedding, out=stream.residual, scale=self.spec.embedding_scale, copies=self.spec.streams,
                                 accumulate=True)
            self.blocks[run.layer].forward(stream, step, caches[position])
            if taps is not None:
                taps.append(stream.total().clone())
        if step.num_logits == 0:
            return None
        hidden = self.final_norm.apply(stream, rows=step.logit_rows)
        logits = ops.linear(hidden, self.lm_head, out_dtype=torch.float32)
        if self.spec.logit_scale != 1.0 or self.spec.logit_softcap is not None:
            ops.logit_transform(logits, self.spec.logit_scale, self.spec.logit_softcap)
        return logits
