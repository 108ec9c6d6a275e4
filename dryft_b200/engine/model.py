"""A decoder put together from a ``ModelSpec``: embedding, the layers' blocks in run order, final
norm and output head.  It is the same class for every architecture; what differs is the spec.

One forward pass serves prefill and decode: it runs exactly the tokens of the step, reads and writes
the cache through each run step's ``CacheEntry``, and returns 32-bit logits at the wanted rows only
(the reference computes the last position only and returns its argmax,
``engine/dryft_qwen3/model.py:185-187,261-262``).
"""

from __future__ import annotations

from typing import List, Optional, Tuple

import torch

from ..cache.store import KVNeed, SequenceCache, StateNeed
from ..config.spec import ModelSpec
from ..parts.base import BLOCKS, EMBEDDINGS, FAMILIES, FFNS, HEADS, MIXERS, NORMS, Residual, Runtime, StepContext


class DecoderModel:
    def __init__(self, spec: ModelSpec, weights, rt: Runtime):
        spec.validate()
        self.spec = spec
        self.rt = rt
        self.vocab_size = spec.vocab_size
        self.hidden_size = spec.hidden_size
        self.embedding = EMBEDDINGS.get(spec.embedding.kind)(spec.embedding.params, spec.embedding_prefix, weights, rt)
        self.blocks = []
        for layer in spec.layers:
            norm_mixer = NORMS.get(layer.norm_mixer.kind)(layer.norm_mixer.params, layer.norm_mixer_prefix, weights, rt)
            mixer = MIXERS.get(layer.mixer.kind)(layer.mixer.params, layer.mixer_prefix, weights, rt)
            norm_ffn = ffn = None
            if layer.ffn is not None:
                if layer.norm_ffn is not None:
                    norm_ffn = NORMS.get(layer.norm_ffn.kind)(layer.norm_ffn.params, layer.norm_ffn_prefix, weights, rt)
                ffn = FFNS.get(layer.ffn.kind)(layer.ffn.params, layer.ffn_prefix, weights, rt)
            extra = {e.name: FAMILIES[e.family].get(e.spec.kind)(e.spec.params, e.prefix, weights, rt) for e in layer.extra}
            make = BLOCKS.get(layer.block)
            self.blocks.append(make(norm_mixer, mixer, norm_ffn, ffn, extra=extra) if extra else make(norm_mixer, mixer, norm_ffn, ffn))
        # a test or a bring-up script may watch the stream: called as layer_tap(run step, block, Residual) after every block
        self.layer_tap = None
        self.final_norm = NORMS.get(spec.final_norm.kind)(spec.final_norm.params, spec.final_norm_prefix, weights, rt)
        self.head = HEADS.get(spec.head.kind)(spec.head.params, spec.head_prefix, weights, rt, embedding=self.embedding)
        # parts between the layers: what a run step is entered through
        self.joints = {j.name: FAMILIES[j.family].get(j.spec.kind)(j.spec.params, j.prefix, weights, rt) for j in spec.joints}
        self.keeps_x0 = any(st.enter is not None for st in spec.schedule)

    # what each run step asks of the cache
    def cache_needs(self) -> Tuple[List[Tuple[Optional[KVNeed], Optional[StateNeed]]], List[Optional[int]]]:
        needs, borrow = [], []
        for st in self.spec.schedule:
            mixer = self.blocks[st.layer].mixer
            needs.append((mixer.kv_need(), mixer.state_need()))
            borrow.append(st.cache_from)
        return needs, borrow

    def named_state_needs(self) -> dict:
        """Per-sequence state of the parts outside the layers: ``{name: StateNeed}`` (today: the embedding's)."""
        need = getattr(self.embedding, "state_need", None)
        need = need() if callable(need) else None
        return {"embedding": need} if need is not None else {}

    def weight_bytes(self) -> int:
        seen, total = set(), 0
        def visit(obj):
            nonlocal total
            for v in vars(obj).values():
                if isinstance(v, torch.Tensor) and v.is_floating_point() and v.dim() >= 1:
                    key = v.data_ptr()
                    if key not in seen:
                        seen.add(key)
                        total += v.numel() * v.element_size()
        visit(self.embedding); visit(self.final_norm); visit(self.head)
        for j in self.joints.values():
            visit(j)
        for b in self.blocks:
            for part in (b.norm_mixer, b.mixer, b.norm_ffn, b.ffn, *getattr(b, "extra", {}).values()):
                if part is not None:
                    visit(part)
        return total

    def forward(self, ctx: StepContext, cache: SequenceCache, want_rows: Optional[torch.Tensor], n_want: int,
                all_rows: bool = False) -> Optional[torch.Tensor]:
        """Run the step's tokens through every run step; logits ``[n_want, vocab]`` float32 at the
        packed rows ``want_rows`` (None if nothing is wanted).  ``all_rows`` says that ``want_rows`` is simply
        every row in order (a decode step), which lets the head take the fused path."""
        if getattr(self.embedding, "takes_state", False):     # an embedding that remembers each sequence's last token
            res = self.embedding.forward(ctx.tokens, ctx.n_tokens, ctx, cache.named_state("embedding"))
        elif getattr(self.embedding, "takes_context", False):   # an embedding that adds the tokens' positions
            res = self.embedding.forward(ctx.tokens, ctx.n_tokens, ctx)
        else:
            res = self.embedding.forward(ctx.tokens, ctx.n_tokens)
        if not isinstance(res, Residual):
            res = Residual(res)
        sched = self.spec.schedule
        x0 = res.x.clone() if self.keeps_x0 else None    # the embedding's output, for the joints that mix it back in
        for i, st in enumerate(sched):
            block = self.blocks[st.layer]
            if st.enter is not None:
                res = self.joints[st.enter[0]].enter(res, x0, st.enter[1], getattr(block, "norm_mixer", None))
            if getattr(block, "takes_next_norms", False):
                # both norms that read the stream next (an arrangement whose mixer and feed-forward read the same stream)
                if i + 1 < len(sched):
                    b = self.blocks[sched[i + 1].layer] if sched[i + 1].enter is None else None
                    nxts = (getattr(b, "norm_mixer", None), getattr(b, "norm_ffn", None) if getattr(b, "takes_next_norms", False) else None)
                else:
                    nxts = (self.final_norm, None)
                res = block.forward(res, ctx, cache.entry(i), cache.state(i), owns_cache=st.cache_from is None, next_norms=nxts)
            elif getattr(block, "takes_next_norm", False):
                # the norm that reads the stream next: the following run step's first norm, or the final norm -- unless a
                # joint transforms the stream in between
                if i + 1 < len(sched):
                    nxt = None if sched[i + 1].enter is not None else getattr(self.blocks[sched[i + 1].layer], "norm_mixer", None)
                else:
                    nxt = self.final_norm
                res = block.forward(res, ctx, cache.entry(i), cache.state(i), owns_cache=st.cache_from is None, next_norm=nxt)
            else:
                res = block.forward(res, ctx, cache.entry(i), cache.state(i), owns_cache=st.cache_from is None)
            if self.layer_tap is not None:
                self.layer_tap(i, block, res)
        if n_want == 0:
            return None
        if res.closer is not None:   # streams that only their block arrangement knows how to join
            return self.head.forward(res.closer.final_rows(res, self.final_norm, want_rows, n_want))
        if (all_rows and res.delta is None and res.ss is not None and hasattr(self.head, "forward_normed")
                and self.head.can_fuse(res.x.shape[0], self.final_norm)):
            xw = res.xw if res.xw_norm is self.final_norm else None
            return self.head.forward_normed(res.x, res.ss, res.ss_parts, self.final_norm, **({"xw": xw} if xw is not None else {}))
        if res.delta is None and res.hn is not None and res.hn_norm is self.final_norm:
            # the kernel that formed the stream left it normed already: only the wanted rows go on
            h = res.hn if all_rows else res.hn.index_select(0, want_rows[:n_want].long())
        elif res.delta is None:
            h = self.final_norm.forward(res.x, rows=want_rows, n_rows=n_want)
        else:
            h = self.final_norm.add_forward(res.x, res.delta, rows=want_rows, n_rows=n_want)
        return self.head.forward(h)
