"""The naive sampler every model offers: no cache, the whole prefix again for each token."""

import torch
import torch.nn.functional as F


class NaiveSampler:
    @torch.inference_mode()
    def generate(self, tokens, max_tokens, temperature=1.0, top_k=None, seed=42):
        """Naive batch-1 streaming sampler that recomputes the whole prefix per token; the
        Engine must agree with it token for token at temperature 0 (reference: gpt.py:526-555)."""
        assert isinstance(tokens, list)
        device = self.get_device()
        rng = None
        if temperature > 0:
            rng = torch.Generator(device=device)
            rng.manual_seed(seed)
        ids = torch.tensor([tokens], dtype=torch.long, device=device)
        for _ in range(max_tokens):
            logits = self.forward(ids)[:, -1, :]
            if top_k is not None and top_k > 0:
                kth, _ = torch.topk(logits, min(top_k, logits.size(-1)))
                logits[logits < kth[:, [-1]]] = -float("inf")
            if temperature > 0:
                probs = F.softmax(logits / temperature, dim=-1)
                nxt = torch.multinomial(probs, num_samples=1, generator=rng)
            else:
                nxt = torch.argmax(logits, dim=-1, keepdim=True)
            ids = torch.cat((ids, nxt), dim=1)
            yield nxt.item()
