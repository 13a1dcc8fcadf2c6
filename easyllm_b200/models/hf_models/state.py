"""What running sequences keep between steps: slots, per-layer caches and states, and the index of one step.

``DecodeState`` is the manager.  A sequence opens a slot, every step appends tokens to some slots, and closing the slot
gives it back; a slot that is used again starts from position 0, which every layer takes as "nothing before".  Each
layer contributes one state object through ``layer.new_state``:

* ``PositionRows``: something for every position, ``[slots, capacity, ...]``, grown in whole blocks of positions; as
  ``KVRows`` keys and values ``[.., kv_heads, dim]``, as ``LatentRows`` one latent and one rotated key part per position;
* ``SlotTensors``: fixed-size tensors per slot (recurrent matrices, last inputs of a short convolution or a token shift);
* a plain dict (the 8-bit cache of Qwen): dense batches of equal length only.

What the embedding keeps (token ids by position, when it looks at the previous token) is one more ``PositionRows``,
``DecodeState.tokens``.  ``DecodeState.step_meta`` is the packed description of one step that the layers read.  All index tensors are built on
the host and copied once; ``DecodeGraph`` replays the one-token step of fixed slots as a CUDA graph, with the positions
advanced on the device.
"""
from __future__ import annotations

import torch

BLOCK = 256          # positions a key/value cache grows by


class PositionRows:
    def __init__(self, slots, capacity, device, **shapes):
        """``name=(shape, dtype)`` per tensor; each becomes an attribute ``[slots, capacity, *shape]``."""
        self.names = list(shapes)
        for name, (shape, dtype) in shapes.items():
            setattr(self, name, torch.zeros(slots, capacity, *shape, dtype=dtype, device=device))

    def grow(self, slots, capacity):
        for name in self.names:
            old = getattr(self, name)
            new = old.new_zeros(slots, capacity, *old.shape[2:])
            new[:old.shape[0], :old.shape[1]] = old
            setattr(self, name, new)


class LatentRows(PositionRows):
    """``c``: per position the normed latent followed by the rotated key part, rows padded to 8 elements."""

    def __init__(self, slots, capacity, rank, rot, device, dtype):
        super().__init__(slots, capacity, device, c=((-(-(rank + rot) // 8) * 8,), dtype))


class KVRows(PositionRows):
    def __init__(self, slots, capacity, kv_heads, dim, vdim, device, dtype):
        super().__init__(slots, capacity, device, k=((kv_heads, dim), dtype), v=((kv_heads, vdim), dtype))

    def load_prefix(self, slots, k, v):
        """Fill positions ``0 .. n`` of ``slots`` with given keys / values ``[n, kv_heads, dim]`` (prefix tuning)."""
        for s in slots:
            self.k[s, :k.shape[0]], self.v[s, :v.shape[0]] = k.to(self.k.dtype), v.to(self.v.dtype)


class SlotTensors:
    def __init__(self, slots, device, **shapes):
        """``name=(shape, dtype)`` per tensor; each becomes an attribute ``[slots, *shape]``."""
        self.names = list(shapes)
        for name, (shape, dtype) in shapes.items():
            setattr(self, name, torch.zeros(slots, *shape, dtype=dtype, device=device))

    def grow(self, slots, capacity):
        for name in self.names:
            old = getattr(self, name)
            new = old.new_zeros(slots, *old.shape[1:])
            new[:old.shape[0]] = old
            setattr(self, name, new)


class DecodeState:
    def __init__(self, model, slots, capacity, device=None, dtype=None):
        w = model.lm_head.weight
        self.device, self.dtype = device or w.device, dtype or w.dtype
        self.capacity = -(-capacity // BLOCK) * BLOCK
        self.layers = [layer.new_state(slots, self.capacity, self.device, self.dtype) for layer in model.model.layers]
        self.tokens = PositionRows(slots, self.capacity, self.device, ids=((), torch.int32)) if model.model.keeps_tokens \
            else None
        self.lengths = [0] * slots
        self.free = list(range(slots - 1, -1, -1))

    @property
    def slots(self):
        return len(self.lengths)

    def open(self):
        """A slot for a new sequence (the manager grows when none is free)."""
        if not self.free:
            n = self.slots
            self._grow(2 * n, self.capacity)
            self.lengths += [0] * n
            self.free = list(range(2 * n - 1, n - 1, -1))
        s = self.free.pop()
        self.lengths[s] = 0
        return s

    def close(self, slot):
        self.lengths[slot] = 0
        self.free.append(slot)

    def reserve(self, length):
        """Room for sequences of ``length`` tokens."""
        if length > self.capacity:
            self._grow(self.slots, -(-max(length, 2 * self.capacity) // BLOCK) * BLOCK)

    def _grow(self, slots, capacity):
        for st in self.layers:
            if not hasattr(st, "grow"):
                raise ValueError("this cache cannot grow: it holds one dense batch of a fixed size")
            st.grow(slots, capacity)
        if self.tokens is not None:
            self.tokens.grow(slots, capacity)
        self.capacity = capacity

    # ---- one step ------------------------------------------------------------------------------
    def step_meta(self, slots, counts, advance=True):
        """Packed meta of a step that appends ``counts[i]`` tokens to ``slots[i]``; the lengths advance."""
        if len(set(slots)) != len(slots) or any(c < 1 for c in counts):
            raise ValueError("a step brings at least one token to each of its (distinct) sequences")
        start = [self.lengths[s] for s in slots]
        self.reserve(max(p + c for p, c in zip(start, counts)))
        dev, S, T = self.device, len(slots), sum(counts)
        cu = [0]
        for c in counts:
            cu.append(cu[-1] + c)
        n = torch.tensor(counts)
        sl, p0 = torch.tensor(slots), torch.tensor(start)
        first = torch.tensor(cu[:-1])
        pos = torch.arange(T) - torch.repeat_interleave(first - p0, n, output_size=T)
        # one host buffer, one copy: sequence borders, slots, start positions | positions, first row of the sequence,
        # row of its first key, keys
        tok_slot = torch.repeat_interleave(sl, n, output_size=T)
        rows = torch.repeat_interleave(first, n, output_size=T)
        buf = torch.cat((torch.tensor(cu), sl, p0, pos, rows, tok_slot * self.capacity, pos + 1)).to(torch.int32)
        if dev.type == "cuda":
            buf = buf.pin_memory().to(dev, non_blocking=True)
        parts = buf.split([S + 1, S, S, T, T, T, T])
        for s, c in zip(slots, counts):
            self.lengths[s] += c if advance else 0
        fresh = not any(start)
        return {"cu_seqlens": parts[0], "seq_slot": parts[1], "seq_pos0": parts[2], "position_ids": parts[3],
                "row_start": parts[4], "kv_base": parts[5], "kv_len": parts[6], "max_seqlen": max(counts),
                "max_position": max(p + c for p, c in zip(start, counts)), "batch": S, "fresh": fresh,
                "one_token": T == S, "kv_capacity": self.capacity,
                "last_rows": torch.tensor(cu[1:]) - 1}


class DecodeGraph:
    """The one-token step of fixed slots as a CUDA graph: embedding, layers, logits and the advance of the positions,
    replayed with new token ids.  The cache must not move while the graph is in use: its capacity is checked, and the
    caller captures anew when the state has grown.  Capturing executes nothing, so no state is touched; run at least one
    eager step before (it initialises the kernels)."""

    def __init__(self, model, state, slots):
        self.state, self.slots, self.capacity = state, list(slots), state.capacity
        self.meta = state.step_meta(slots, [1] * len(slots), advance=False)
        # host-side bounds that hold for every replay
        self.meta.update(max_position=state.capacity, kv_bound=state.capacity, fresh=False, one_token=True)
        self.ids = torch.zeros(len(slots), dtype=torch.long, device=state.device)
        model.prepare_positions(state.capacity, state.device)
        self.graph = torch.cuda.CUDAGraph()
        torch.cuda.synchronize()
        with torch.no_grad(), torch.cuda.graph(self.graph):
            self.logits = model.logits(model.hidden_states(self.ids, self.meta, state.layers, tokens=state.tokens))
            for name in ("seq_pos0", "position_ids", "kv_len"):
                self.meta[name].add_(1)

    def step(self, tokens):
        """fp32 logits ``[n, vocab]`` after ``tokens [n]`` (a buffer the next step overwrites)."""
        st = self.state
        if st.capacity != self.capacity or any(st.lengths[s] >= self.capacity for s in self.slots):
            raise RuntimeError("the cache moved or is full: capture the decode step again")
        self.ids.copy_(tokens)
        self.graph.replay()
        for s in self.slots:
            st.lengths[s] += 1
        return self.logits
