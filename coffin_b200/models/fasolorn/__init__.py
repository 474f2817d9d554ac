"""Fasolorn: windowed attention with sinks and mixed values, windowed latent attention, routed feed-forwards with identity experts."""
