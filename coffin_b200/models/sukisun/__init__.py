"""Sukisun: depth-averaged residual, latent attention with shared caches, Mamba-2."""
