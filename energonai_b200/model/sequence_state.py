"""What a batch of sequences holds between steps, for the decoders put together from a list of layers:
one entry per layer that keeps something, and where each sequence begins and stands.

An entry is a RingCache (rows of past positions, all of them or a window) or a RecurrentState (a fixed
amount per sequence); both are prepared for a new batch, can give up or split off sequences, and tell
how many positions they have room for."""
import torch

from .attention import KVCache


def round_up(n, m):
    return -(-n // m) * m


class RingCache(KVCache):
    """[batch, keep + rows, width]: `keep` rows for the first positions of each sequence, if a window keeps them
    visible, and a ring in which position p lives in row p mod rows.  `window` is the longest window of
    the layers that read it (0: unlimited), so rows = min(positions, window).  A ring shorter than its
    window has never wrapped, which is why it can grow like a KVCache."""

    def __init__(self, width, window=0, reserve=256, keep=0):
        super().__init__(reserve)
        self.width, self.window, self.kept = width, window, keep

    def rows_for(self, positions):
        return self.kept + (min(positions, self.window) if self.window > 0 else positions)

    def prepare(self, batch, positions, dtype, device):
        """For a new batch: room for `positions`; memory kept from an earlier batch of the same size
        is used again when it has exactly the rows that are needed."""
        self.reset()
        rows = self.rows_for(positions)
        if self.buf is None or self.buf.shape[:2] != (batch, rows) or self.buf.dtype != dtype or self.buf.device != device:
            self.buf = torch.zeros((batch, rows, self.width), dtype=dtype, device=device)     # (unwritten rows must be finite)

    def grow(self, positions):
        rows = self.rows_for(positions)
        have = self.buf.shape[1]
        if rows > have:
            old = self.buf
            self.buf = torch.zeros((old.shape[0], self.rows_for(positions + self.reserve), self.width), dtype=old.dtype, device=old.device)
            self.buf[:, :have] = old

    def keep(self, rows):
        self.buf = self.buf.index_select(0, rows)

    def fork(self):
        """The same memory under another owner (which then keeps its own sequences)."""
        out = RingCache(self.width, self.window, self.reserve, self.kept)
        out.buf, out.len = self.buf, self.len
        return out

    def room(self):
        """Positions it can take; None if it holds its whole window."""
        rows = self.buf.shape[1] - self.kept
        return rows if self.window <= 0 or rows < self.window else None

    def pointers(self):
        return (self.buf.data_ptr(),)


class RecurrentState:
    """fp32 tensors (or of another type) [batch, ...] that a recurrent layer carries from token to token;
    `shapes` gives each one's size per sequence.  A new batch starts from zero."""

    def __init__(self, shapes, dtype=torch.float32):
        self.shapes, self.dtype, self.tensors, self.len = [tuple(s) for s in shapes], dtype, None, 0

    def prepare(self, batch, positions, dtype, device):
        t = self.tensors
        if t is None or t[0].shape[0] != batch or t[0].device != device:
            self.tensors = [torch.zeros((batch,) + s, dtype=self.dtype, device=device) for s in self.shapes]
        else:
            for x in t:
                x.zero_()
        self.len = 0

    def grow(self, positions):
        pass

    def keep(self, rows):
        self.tensors = [t.index_select(0, rows) for t in self.tensors]

    def fork(self):
        out = RecurrentState(self.shapes, self.dtype)
        out.tensors, out.len = self.tensors, self.len
        return out

    def room(self):
        return None

    def pointers(self):
        return tuple(t.data_ptr() for t in self.tensors)


class SequenceState:
    """What a batch of sequences holds between steps: the caches, where each sequence begins in the
    left-padded batch, and the common position.  `kv_state` = (position of the next token, its
    successor) lives on the device, where captured steps advance it."""

    def __init__(self, caches):
        self.caches = caches                    # {layer, or (layer, part): RingCache or RecurrentState}
        self.first = self.kv_state = None
        self.batch, self.length, self.padded = 0, 0, False

    def begin(self, first, prompt_len, reserve, dtype, device):
        """first: list with the number of padding positions in front of each sequence."""
        B = len(first)
        if self.first is None or self.first.numel() != B or self.first.device != device:
            self.first = torch.empty(B, dtype=torch.int32, device=device)
            self.kv_state = torch.empty(2, dtype=torch.int32, device=device)
        self.first.copy_(torch.tensor(first, dtype=torch.int32))
        self.kv_state.copy_(torch.tensor([prompt_len, prompt_len + 1], dtype=torch.int32))
        self.batch, self.length, self.padded = B, prompt_len, any(first)
        for c in self.caches.values():
            c.prepare(B, prompt_len + max(0, reserve), dtype, device)
            c.len = prompt_len

    def ensure(self, positions):
        for c in self.caches.values():
            c.grow(positions)

    def capacity(self):
        """Positions the caches can take; None if there is no limit."""
        caps = [r for r in (c.room() for c in self.caches.values()) if r is not None]
        return min(caps) if caps else None

    def set_length(self, n):
        self.length = n
        for c in self.caches.values():
            c.len = n

    def advance(self):
        self.kv_state.add_(1)
        self.set_length(self.length + 1)

    def keep(self, rows):
        """Only the sequences `rows` (list of indices) go on; the memory of the others is given back."""
        if list(rows) == list(range(self.batch)):
            return
        sel = torch.tensor(list(rows), dtype=torch.long, device=self.first.device)
        self.first = self.first.index_select(0, sel)
        for c in self.caches.values():
            c.keep(sel)
        self.batch = len(rows)

    def fork(self, rows):
        """A state of its own for the sequences `rows`."""
        out = SequenceState({k: c.fork() for k, c in self.caches.items()})
        out.first, out.kv_state = self.first, self.kv_state.clone()
        out.batch, out.length, out.padded = self.batch, self.length, self.padded
        if list(rows) == list(range(self.batch)):
            raise RuntimeError("fork: nothing would be left")
        out.keep(rows)
        return out


class PromptContext:
    is_prompt = True
    """One prompt pass: shapes, padding, and what the layers run so far left for later ones."""

    def __init__(self, state, batch, seq, mask):
        self.state, self.batch, self.seq, self.mask = state, batch, seq, mask
        self.first = state.first if state.padded else None
        self.pos = None                         # positions start at 0
        self.latents = {}


class StepContext:
    is_prompt = False
    """One generation step."""

    def __init__(self, state):
        self.state, self.batch = state, state.batch
        self.first = state.first if state.padded else None
        self.seq = 1
        self.pos = state.kv_state[0:1]
