"""Paged batches for the kernel tests of layered decoders: scattered blocks, arbitrary (past, new) lengths."""
import torch


class PagedBatch:
    """``spans``: (past, new) of every sequence. Blocks are handed out in random order from a pool with spare ones."""

    def __init__(self, spans, block_size=16, seed=0, device="cuda"):
        g = torch.Generator().manual_seed(seed)
        self.spans, self.bs, self.device = spans, block_size, device
        self.B, self.T = len(spans), sum(n for _, n in spans)
        need = [(p + n + block_size - 1) // block_size for p, n in spans]
        self.num_blocks = sum(need) + 5
        order = torch.randperm(self.num_blocks, generator=g).tolist()
        self.tables = []
        for k in need:
            self.tables.append(order[:k])
            order = order[k:]
        i32 = lambda v: torch.tensor(v, dtype=torch.int32, device=device)
        begins, blocks = [0], [0]
        for (p, n), t in zip(spans, self.tables):
            begins.append(begins[-1] + n)
            blocks.append(blocks[-1] + len(t))
        self.begins = begins
        self.positions = i32([p + j for p, n in spans for j in range(n)])
        self.slot_map = i32([self.slot(b, p + j) for b, (p, n) in enumerate(spans) for j in range(n)])
        self.args = dict(past_lens=i32([p for p, _ in spans]), subsequence_begins=i32(begins), block_indices=i32([x for t in self.tables for x in t]),
                         block_indices_begins=i32(blocks), B=self.B, T=self.T, block_size=block_size)
        self.max_q_len = max(n for _, n in spans)
        self.max_ctx = max(p + n for p, n in spans)

    def slot(self, b, pos):
        return self.tables[b][pos // self.bs] * self.bs + pos % self.bs

    def fill(self, per_seq, pitch, dtype):
        """per_seq: [past + new, heads, D] of every sequence -> cache [blocks, heads, block_size, pitch] (padding zero)."""
        heads, D = per_seq[0].shape[1:]
        cache = torch.zeros((self.num_blocks, heads, self.bs, pitch), dtype=dtype, device=self.device)
        for b, x in enumerate(per_seq):
            for pos in range(x.shape[0]):
                s = self.slot(b, pos)
                cache[s // self.bs, :, s % self.bs, :D] = x[pos].to(dtype)
        return cache
