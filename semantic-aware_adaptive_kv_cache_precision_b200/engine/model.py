"""A decoder model built from a `ModelSpec`: embedding, blocks in their run
order, final norm, output head. It owns no sizes of its own: everything comes
from the spec, and every block is built from its part specs through the part
registry. The forward pass is the reference's `Model.run`
(`src/microinfer/model.py:345-403`) over a batch of sequences."""

from __future__ import annotations

import torch

from .. import ops
from ..cache.needs import StateNeed
from ..parts import build_part
from ..weights import TensorDecl, load_checkpoint, random_arena


class DecoderModel:
    def __init__(self, spec, mode: str = "bfloat16", device="cuda"):
        if mode not in ("bfloat16", "float32"):
            raise ValueError(f"dtype must be 'bfloat16' or 'float32', got {mode!r}")
        self.spec, self.mode, self.device = spec, mode, torch.device(device)
        self.act_dtype = torch.float32 if mode == "float32" else torch.bfloat16
        self.blocks = [build_part(b, b.prefix, mode) for b in spec.blocks]
        self.final_norm = build_part(spec.final_norm, _strip(spec.final_norm_name), mode)
        owners = {}
        for call in spec.run_order:
            if not 0 <= call.block < len(self.blocks):
                raise ValueError(f"run order names block {call.block}, the model has "
                                 f"{len(self.blocks)}")
            owners.setdefault(call.cache, call.block)
        if sorted(owners) != list(range(len(owners))):
            raise ValueError("cache entries of the run order must be numbered 0, 1, 2, ...")
        if spec.bigram and spec.position_name:
            raise ValueError("a table of pairs beside learned positions is not built")
        self._owners = owners
        self.arena = None
        #: whether every part says its step can be captured in a CUDA graph
        self.graph_safe = all(getattr(b, "graph_safe", True) for b in self.blocks)

    # -- tensors ----------------------------------------------------------------

    def tensor_decls(self) -> list[TensorDecl]:
        spec = self.spec
        decls = [TensorDecl(spec.embed_name, (spec.vocab_size, spec.hidden))]
        if spec.position_name:
            decls.append(TensorDecl(spec.position_name, (spec.max_positions, spec.hidden)))
        if spec.bigram:
            decls.append(TensorDecl(spec.bigram.name, (spec.bigram.buckets + 1, spec.hidden)))
        for block in self.blocks:
            decls += block.tensor_decls()
        decls += self.final_norm.tensor_decls()
        if spec.input_mix_name:
            decls.append(TensorDecl(spec.input_mix_name, (spec.hidden, 2 * spec.hidden)))
        if not spec.tie_head:
            decls.append(TensorDecl(spec.head_name, (spec.vocab_size, spec.hidden)))
        if spec.head_bias_name:
            decls.append(TensorDecl(spec.head_bias_name, (spec.vocab_size,), init="zeros"))
        return decls

    @staticmethod
    def tensor_decls_of(spec) -> list[TensorDecl]:
        """The declarations without a device (for writing random checkpoints)."""
        return DecoderModel(spec, "float32", "cpu").tensor_decls()

    def load(self, folder) -> None:
        self._bind(load_checkpoint(folder, self.tensor_decls(), self.mode, self.device,
                                   ignore=self.spec.ignore_tensors))

    def load_random(self, seed: int) -> None:
        self._bind(random_arena(self.tensor_decls(), seed, self.spec.init_std, self.mode,
                                self.device, self.spec.stored_dtype))

    def _bind(self, arena) -> None:
        self.embed = arena.view(self.spec.embed_name)
        self.head = self.embed if self.spec.tie_head else arena.view(self.spec.head_name)
        self.head_bias = arena.view(self.spec.head_bias_name) if self.spec.head_bias_name else None
        self.positions = arena.view(self.spec.position_name) if self.spec.position_name else None
        self.pairs = arena.view(self.spec.bigram.name) if self.spec.bigram else None
        self.input_mix = arena.view(self.spec.input_mix_name) if self.spec.input_mix_name else None
        for block in self.blocks:
            block.bind(arena)
        self.final_norm.bind(arena)
        self.arena = arena

    def kernel_libraries(self) -> list:
        """The kernel libraries this model's steps launch, as far as its parts name them."""
        names = ["elementwise", "sampling"]
        for block in list(self.blocks) + [self.final_norm]:
            names += list(getattr(block, "kernel_libraries", ()))
        return list(dict.fromkeys(names))

    @property
    def weight_bytes(self) -> int:
        return 0 if self.arena is None else self.arena.nbytes

    # -- cache ------------------------------------------------------------------

    def cache_needs(self) -> list:
        """What each cache entry must hold: the need of the block that owns it; behind the blocks'
        entries, where the embedding reads pairs of tokens, the token a sequence brought last."""
        needs = [self.blocks[self._owners[e]].cache_need() for e in range(len(self._owners))]
        return needs + ([StateNeed((1,), "int32")] if self.spec.bigram else [])

    def prepare(self, max_positions: int) -> None:
        for block in self.blocks:
            block.prepare(self.device, max_positions)

    # -- the forward pass ---------------------------------------------------------

    def hidden(self, step, cache, capture: list | None = None) -> torch.Tensor:
        """The residual stream [T, hidden] (fp32) after the last layer call; the
        cache entries that the calls own are extended by the step's tokens.

        With `capture` (a list), copies of the stream are appended to it: after the
        embedding and after every layer call but the last, the order in which the
        reference captures hidden states (`src/microinfer/model.py:355-364, 398-402`);
        `final_states` gives the entry that closes that list."""
        if self.arena is None:
            raise RuntimeError("no weights on the device; load a checkpoint first")
        streams = getattr(self.spec, "streams", 1)
        if streams > 1:          # every stream starts as the embedding's output
            x = torch.empty((streams, step.tokens, self.spec.hidden), dtype=torch.float32,
                            device=self.device)
            self._embed(step, cache, x[0])
            ops.streams_spread(x)
        else:
            x = self._embed(step, cache)

        def stream(x):           # what the streams stand for: their sum
            return ops.streams_step(x, reduce=True) if x.dim() == 3 else x.clone()

        if capture is not None:
            capture.append(stream(x))
        # calls with `mix_input` replace the stream by W [x; x0]: the two halves of the
        # product's input lie side by side, the embedding's output in the second for good
        both = None
        if self.input_mix is not None and any(c.mix_input for c in self.spec.run_order):
            if streams > 1:
                raise ValueError("the input mix is not built for several streams")
            both = torch.empty((step.tokens, 2 * self.spec.hidden), dtype=self.act_dtype,
                               device=self.device)
            both[:, self.spec.hidden:].copy_(x)
        written = set()
        pending = None          # a block's last output, not yet added to the stream
        last = len(self.spec.run_order) - 1
        for i, call in enumerate(self.spec.run_order):
            view = cache.entry_view(call.cache, step.tables)
            block = self.blocks[call.block]
            if call.mix_input and both is not None:
                if pending is not None:
                    _settle(x, pending)
                    pending = None
                both[:, :self.spec.hidden].copy_(x)
                x = ops.linear(both, self.input_mix, out_dtype=torch.float32)
            if getattr(block, "carries_pending", False):
                pending = block.forward(x, step, view, call.cache not in written, pending,
                                        leave_pending=i < last and capture is None)
            else:
                if pending is not None:
                    _settle(x, pending)
                block.forward(x, step, view, call.cache not in written)
                pending = None
            written.add(call.cache)
            if capture is not None and i < last:
                capture.append(stream(x))
        if pending is not None:
            _settle(x, pending)
        return ops.streams_step(x, reduce=True) if x.dim() == 3 else x

    def _embed(self, step, cache, out=None) -> torch.Tensor:
        """The stream at the start: the tokens' rows of the embedding times its scale, plus
        the learned vectors of their positions, or the rows of a table of pairs of tokens, where
        the model has them."""
        if self.pairs is not None:
            last = cache.entry_view(len(self._owners), step.tables).state
            b = self.spec.bigram
            return ops.embed_pairs(step, self.embed, self.pairs, b.mul_prev, b.mul_cur, last,
                                   out=out, scale=self.spec.embed_scale)
        if self.positions is not None and step.max_position >= self.positions.shape[0]:
            raise ValueError(f"position {step.max_position} is beyond the model's "
                             f"{self.positions.shape[0]} learned positions")
        return ops.embed(step.token_ids, self.embed, out=out, scale=self.spec.embed_scale,
                         positions=step.positions, position_table=self.positions)

    def final_states(self, x: torch.Tensor) -> torch.Tensor:
        """The stream after the final norm, fp32 [T, hidden]: the last entry of the captured
        hidden states."""
        return self.final_norm.forward(x, out_dtype=torch.float32)

    def logits(self, x: torch.Tensor, rows: torch.Tensor) -> torch.Tensor:
        """fp32 logits [len(rows), vocab] of the token rows `rows` of `x`: only
        these rows go through the final norm and the output head."""
        normed = self.final_norm.forward(x, rows=rows)
        out = ops.linear(normed, self.head, self.head_bias, out_dtype=torch.float32)
        if self.spec.logit_scale != 1.0 or self.spec.logit_softcap:
            ops.scale_cap_(out, self.spec.logit_scale, self.spec.logit_softcap)
        return out


def _settle(x, pending) -> None:
    """Add what a block left pending: a plain fp32 delta, or an update that knows how it
    goes into the streams."""
    if hasattr(pending, "apply"):
        pending.apply(x)
    else:
        ops.add_into(x, pending)


def _strip(name: str) -> str:
    return name[:-len(".weight")] if name.endswith(".weight") else name
